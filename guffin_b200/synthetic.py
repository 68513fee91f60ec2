"""Seeded synthetic GGUF-format weights, activations and model geometries.

Stands in for the real Gemma checkpoints (none ship with this repository): tensors take the
shapes, block formats and value distributions of the workloads the benchmarks name, all from a
numpy PCG64 seed so the CPU oracle and the CUDA path see identical bytes.

Block formats follow the reference's definitions (src/tensor/quantization.cpp:430-593):
Q8_0 = f16 d + 32 int8; Q4_K = f16 d, f16 dmin, 12 packed 6-bit scale/min bytes, 128 nibble
bytes; Q6_K = 128 low-nibble bytes, 64 high-bit bytes, 16 int8 scales, f16 d.
"""
from __future__ import annotations

import math

import numpy as np

Q8_0, Q4_K, Q6_K = 8, 12, 14
BLOCK_ELEMENTS = {Q8_0: 32, Q4_K: 256, Q6_K: 256}
BLOCK_BYTES = {Q8_0: 34, Q4_K: 144, Q6_K: 210}


def _positive_f16(rng: np.random.Generator, count: int, sigma: float) -> np.ndarray:
    values = np.abs(rng.normal(0.0, sigma, count)).astype(np.float16)
    values[values == 0] = max(np.float16(sigma), np.float16(6e-8))
    return values.view(np.uint8).reshape(count, 2)


def q4k_blocks(rng, count: int, sigma: float = 1e-3) -> np.ndarray:
    """d, dmin ~ |N(0, sigma)|; every 6-bit scale/min field uniform in [0, 63] (uniform bytes
    make all sixteen packed fields uniform); nibbles uniform in [0, 15]."""
    blocks = rng.integers(0, 256, (count, 144), dtype=np.uint8)
    blocks[:, 0:2] = _positive_f16(rng, count, sigma)
    blocks[:, 2:4] = _positive_f16(rng, count, sigma)
    return blocks


def q6k_blocks(rng, count: int, sigma: float = 1e-3) -> np.ndarray:
    """6-bit quants uniform; int8 sub-scales uniform in [-64, 63]; d ~ |N(0, sigma)|."""
    blocks = rng.integers(0, 256, (count, 210), dtype=np.uint8)
    blocks[:, 192:208] = rng.integers(-64, 64, (count, 16), dtype=np.int8).view(np.uint8)
    blocks[:, 208:210] = _positive_f16(rng, count, sigma)
    return blocks


def q80_blocks(rng, count: int, sigma: float = 1e-2) -> np.ndarray:
    """f16 scale ~ |N(0, sigma)|; int8 uniform in [-127, 127]."""
    blocks = np.empty((count, 34), np.uint8)
    blocks[:, 0:2] = _positive_f16(rng, count, sigma)
    blocks[:, 2:] = rng.integers(-127, 128, (count, 32), dtype=np.int8).view(np.uint8)
    return blocks


_MAKERS = {Q4_K: q4k_blocks, Q6_K: q6k_blocks, Q8_0: q80_blocks}


def make_weight(rng, dtype: int, k: int, n: int, sigma: float | None = None) -> np.ndarray:
    """Native GGUF payload of a [K, N] projection: column n owns K/block consecutive blocks."""
    assert k % BLOCK_ELEMENTS[dtype] == 0
    count = n * (k // BLOCK_ELEMENTS[dtype])
    blocks = _MAKERS[dtype](rng, count) if sigma is None else _MAKERS[dtype](rng, count, sigma)
    return blocks.reshape(-1)


def weight_bytes(dtype: int, k: int, n: int) -> int:
    return n * (k // BLOCK_ELEMENTS[dtype]) * BLOCK_BYTES[dtype]


# ---------------------------------------------------------------------------- geometries

def _config(hidden, ffn, heads, kv_heads, head_dim, layers, vocab, window, pattern,
            base_g, scale_g, base_l, scale_l, attn_cap, final_cap, qk_norm, kv_f16):
    return dict(hidden=hidden, ffn=ffn, heads=heads, kv_heads=kv_heads, head_dim=head_dim,
                layers=layers, vocab=vocab, sliding_window=window, sliding_pattern=pattern,
                rope_base_global=base_g, rope_scale_global=scale_g, rope_base_local=base_l,
                rope_scale_local=scale_l, rms_eps=1e-6, attn_softcap=attn_cap,
                final_softcap=final_cap, uses_qk_norm=qk_norm, kv_f16=kv_f16,
                attention_scale=1.0 / math.sqrt(head_dim))


def model_config(name: str) -> dict:
    """Geometries of the reference's three models (scripts/gemma3_target_reference.py:28-29,
    scripts/gemma3_reference_golden.py:41-42, tests/reference/gemma2_reference.cpp) and small
    same-shaped stand-ins for tests."""
    if name == "gemma3-12b":      # target: F16 KV, global RoPE 1e6 scaled by 1/8, local 1e4
        return _config(3840, 15360, 16, 8, 256, 48, 262144, 1024, 6, 1e6, 0.125, 1e4, 1.0, 0.0, 0.0, 1, 1)
    if name == "gemma3-270m":     # drafter: F32 KV, unscaled global RoPE
        return _config(640, 2048, 4, 1, 256, 18, 262144, 512, 6, 1e6, 1.0, 1e4, 1.0, 0.0, 0.0, 1, 0)
    if name == "gemma2-9b":
        return _config(3584, 14336, 16, 8, 256, 42, 256000, 4096, 2, 1e4, 1.0, 1e4, 1.0, 50.0, 30.0, 0, 1)
    if name == "tiny-target":     # 12B block shape shrunk: 7 layers cover a local and a global layer
        return _config(512, 1024, 4, 2, 256, 7, 2048, 16, 6, 1e6, 0.125, 1e4, 1.0, 0.0, 0.0, 1, 1)
    if name == "tiny-draft":
        return _config(256, 512, 4, 1, 256, 6, 2048, 8, 6, 1e6, 1.0, 1e4, 1.0, 0.0, 0.0, 1, 0)
    if name == "tiny-gemma2":
        return _config(512, 1024, 4, 2, 256, 4, 2048, 16, 2, 1e4, 1.0, 1e4, 1.0, 50.0, 30.0, 0, 1)
    raise KeyError(name)


def use_more_bits(layer: int, layers: int) -> bool:
    """Which layers a Q4_K_M file stores attn_v / ffn_down in Q6_K: the published llama.cpp
    quantiser rule (first and last eighth, and every third layer between), which yields 24 of
    48 layers for the 12B model as the reference's byte accounting reports."""
    return layer < layers // 8 or layer >= 7 * layers // 8 or (layer - layers // 8) % 3 == 2


def tensor_types(name: str, config: dict) -> dict:
    """Per-tensor GGUF dtype for each model family."""
    types = {}
    L = config["layers"]
    for l in range(L):
        for t in ("attn_q", "attn_k", "attn_v", "attn_output", "ffn_gate", "ffn_up", "ffn_down"):
            if name.endswith("270m") or name == "tiny-draft":
                dtype = Q8_0
            elif name.startswith("gemma2") or name == "tiny-gemma2":
                dtype = Q4_K
            else:
                dtype = Q6_K if t in ("attn_v", "ffn_down") and use_more_bits(l, L) else Q4_K
            types[f"blk.{l}.{t}.weight"] = dtype
    if name.endswith("270m") or name == "tiny-draft":
        types["token_embd.weight"] = Q8_0
    elif name.startswith("gemma2") or name == "tiny-gemma2":
        types["token_embd.weight"] = Q6_K     # embedding rows
        types["output.weight"] = Q8_0         # separate Q8_0 head (gemma2_metal_plan.cpp:495-512)
    else:
        types["token_embd.weight"] = Q6_K
    return types


def matrix_shapes(config: dict) -> dict:
    H, F, hd = config["hidden"], config["ffn"], config["head_dim"]
    q, kv = config["heads"] * hd, config["kv_heads"] * hd
    return {"attn_q": (H, q), "attn_k": (H, kv), "attn_v": (H, kv), "attn_output": (q, H),
            "ffn_gate": (H, F), "ffn_up": (H, F), "ffn_down": (F, H)}


def iter_model_weights(name: str, seed: int, config: dict | None = None):
    """Yields (GGUF tensor name, value) one tensor at a time: value is (dtype, K, N, uint8 payload)
    for matrices and a float32 array for norm vectors.  Lets a loader upload a 12B model without
    holding all of it in host memory."""
    config = config or model_config(name)
    rng = np.random.default_rng(seed)
    types = tensor_types(name, config)
    shapes = matrix_shapes(config)
    H, V = config["hidden"], config["vocab"]

    def gamma(n):
        return (1.0 + 0.1 * rng.standard_normal(n)).astype(np.float32)

    # Embedding / head blocks are scaled so that an embedded token has unit RMS after the
    # sqrt(hidden) factor, as trained checkpoints roughly do; otherwise a random tied model just
    # echoes its input token and every proposal is trivially accepted.
    def table_sigma(dtype):
        code_rms = {Q6_K: 685.0, Q8_0: 73.3, Q4_K: 300.0}[dtype]
        return 1.0 / (code_rms * math.sqrt(H))

    embd_type = types["token_embd.weight"]
    yield "token_embd.weight", (embd_type, H, V, make_weight(rng, embd_type, H, V, table_sigma(embd_type)))
    if "output.weight" in types:
        head_type = types["output.weight"]
        yield "output.weight", (head_type, H, V, make_weight(rng, head_type, H, V, table_sigma(head_type)))
    yield "output_norm.weight", gamma(H)
    for l in range(config["layers"]):
        for t, (k, n) in shapes.items():
            key = f"blk.{l}.{t}.weight"
            yield key, (types[key], k, n, make_weight(rng, types[key], k, n))
        for t in ("attn_norm", "post_attention_norm", "ffn_norm", "post_ffw_norm"):
            yield f"blk.{l}.{t}.weight", gamma(H)
        if config["uses_qk_norm"]:
            yield f"blk.{l}.attn_q_norm.weight", gamma(config["head_dim"])
            yield f"blk.{l}.attn_k_norm.weight", gamma(config["head_dim"])


def make_model_weights(name: str, seed: int, config: dict | None = None) -> dict:
    """All tensors of iter_model_weights in one dict."""
    return dict(iter_model_weights(name, seed, config))


# ---------------------------------------------------------------------------- layered models

def zasevik_config(width, layers, heads, dim, vdim, rank, vocab, mlps, eps=1e-6) -> dict:
    """A Zasevik configuration with one attention geometry; layer i takes mlps[i % len(mlps)] (dense_mlp / expert_mlp / None)."""
    mixer = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=1.0 / math.sqrt(dim))
    return dict(architecture="Zasevik", embedding=dict(scale=math.sqrt(width)), norm=dict(eps=eps), vocab=vocab, width=width,
                layers=[dict(type="latent_attention", mixer=dict(mixer), mlp=mlps[i % len(mlps)]) for i in range(layers)])


def dense_mlp(ff) -> dict:
    return dict(kind="dense", ff=ff)


def expert_mlp(ff, experts, top, limit, shared_ff=0, shared_limit=0.0) -> dict:
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if shared_ff:
        mlp["shared"] = dict(ff=shared_ff, limit=shared_limit)
    return mlp


def zasevik_shapes(config: dict) -> dict:
    """Tensor name -> shape of every tensor of a Zasevik configuration."""
    W, shapes = config["width"], {"embed": (config["vocab"], config["width"]), "final.norm": (config["width"],)}
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer.get("mlp")
        H, R = m["heads"], m["kv_rank"]
        shapes.update({f"{p}.norm1": (W,), f"{p}.norm1b": (W,), f"{p}.ls1": (W,), f"{p}.mix.q": (H * m["dim"], W), f"{p}.mix.dkv": (R, W),
                       f"{p}.mix.dkv.norm": (R,), f"{p}.mix.uk": (H * m["dim"], R), f"{p}.mix.uv": (H * m["vdim"], R), f"{p}.mix.sink": (H,),
                       f"{p}.mix.o": (W, H * m["vdim"])})
        if not f:
            continue
        shapes.update({f"{p}.norm2": (W,), f"{p}.norm2b": (W,), f"{p}.ls2": (W,)})
        if f["kind"] == "dense":
            shapes.update({f"{p}.mlp.up": (f["ff"], W), f"{p}.mlp.down": (W, f["ff"])})
            continue
        for e in range(f["router"]["experts"]):
            shapes.update({f"{p}.mlp.e{e}.gate": (f["expert"]["ff"], W), f"{p}.mlp.e{e}.up": (f["expert"]["ff"], W), f"{p}.mlp.e{e}.down": (W, f["expert"]["ff"])})
        shapes[f"{p}.mlp.router"] = (f["router"]["experts"], W)
        if f.get("shared"):
            ff = f["shared"]["ff"]
            shapes.update({f"{p}.mlp.shared.gate": (ff, W), f"{p}.mlp.shared.up": (ff, W), f"{p}.mlp.shared.down": (W, ff), f"{p}.mlp.shared.sg": (1, W)})
    return shapes


def iter_zasevik_weights(config: dict, seed: int):
    """Yields (name, array): matrices as bfloat16 bits with entries of variance 1 / inputs, vectors as f32."""
    rng = np.random.default_rng(seed)
    for name, shape in zasevik_shapes(config).items():
        if len(shape) == 2:
            values = rng.standard_normal(shape, dtype=np.float32) * np.float32(1.0 / math.sqrt(shape[1]))
            bits = values.view(np.uint32)
            yield name, ((bits + 0x7fff + ((bits >> 16) & 1)) >> 16).astype(np.uint16)
        elif name.endswith(".sink"):
            yield name, rng.normal(1.0, 1.0, shape).astype(np.float32)
        elif ".ls" in name or name.endswith("dkv.norm"):
            yield name, rng.uniform(0.5, 1.5, shape).astype(np.float32)
        else:
            yield name, rng.normal(0.0, 0.2, shape).astype(np.float32)


def zasevik_active_parameters(config: dict) -> int:
    """Matrix elements one token's pass multiplies with (chosen experts only; the head included)."""
    total = 0
    for name, shape in zasevik_shapes(config).items():
        if len(shape) != 2:
            continue
        parts, share = name.split("."), 1.0
        if len(parts) > 2 and parts[1] == "mlp" and parts[2][0] == "e" and parts[2][1:].isdigit():
            router = config["layers"][int(parts[0][1:])]["mlp"]["router"]
            share = router["top"] / router["experts"]
        total += share * shape[0] * shape[1]
    return int(round(total))


def tufirax_attention(heads, kv_heads, dim, scale=None, softcap=30.0, rot_dims=None, base=10000.0, ff=0, weights_of=None) -> dict:
    """A layer of grouped-query attention and a gated feed-forward (none with ff = 0)."""
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=1.0 / math.sqrt(dim) if scale is None else scale, softcap=softcap,
                 rot=dict(base=base, dims=dim if rot_dims is None else rot_dims))
    return _tufirax_layer("attention", mixer, ff, weights_of)


def tufirax_state_space(heads, vdim, state, groups=1, conv=4, norm_groups=1, ff=0, weights_of=None) -> dict:
    """A state-space layer and a gated feed-forward (none with ff = 0)."""
    return _tufirax_layer("mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups), ff, weights_of)


def _tufirax_layer(kind, mixer, ff, weights_of) -> dict:
    layer = dict(type=kind, mixer=mixer, mlp=dense_mlp(ff) if ff else None)
    return layer if weights_of is None else dict(layer, weights_of=weights_of)


def tufirax_config(width, vocab, layers, eps=1e-6) -> dict:
    return dict(architecture="Tufirax", norm=dict(eps=eps), vocab=vocab, width=width, layers=layers)


def tufirax_shapes(config: dict) -> dict:
    """Tensor name -> shape of every tensor of a Tufirax configuration."""
    W, shapes = config["width"], {"embed": (config["vocab"], config["width"])}
    for i, layer in enumerate(config["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}", layer["mixer"]
        inner = m["heads"] * m["vdim"]
        shapes[f"{p}.norm1"] = (W,)
        if layer["type"] == "attention":
            q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            shapes.update({f"{p}.mix.q": (q, W), f"{p}.mix.k": (k, W), f"{p}.mix.q.norm": (q,), f"{p}.mix.k.norm": (k,), f"{p}.mix.sink": (m["heads"],),
                           f"{p}.mix.g": (m["heads"], W)})
        else:
            channels = inner + 2 * m["groups"] * m["state"]
            shapes.update({f"{p}.mix.in": (inner + channels + m["heads"], W), f"{p}.mix.conv": (channels, m["conv"]), f"{p}.mix.conv.b": (channels,),
                           f"{p}.mix.dt_bias": (m["heads"],), f"{p}.mix.A_log": (m["heads"],), f"{p}.mix.D": (m["heads"],), f"{p}.mix.norm": (inner,)})
        shapes[f"{p}.mix.o"] = (W, inner)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            shapes.update({f"{p}.norm2": (W,), f"{p}.mlp.gate": (ff, W), f"{p}.mlp.up": (ff, W), f"{p}.mlp.down": (W, ff)})
    shapes.update({"final.norm": (W,), "head": (config["vocab"], W)})
    return shapes


def iter_tufirax_weights(config: dict, seed: int):
    """Yields (name, array): matrices as bfloat16 bits with entries of variance 1 / inputs (the token table's 1), vectors
    as f32.  Step sizes lie between 0.001 and 0.3, decay rates between 1 and 16."""
    rng = np.random.default_rng(seed)
    for name, shape in tufirax_shapes(config).items():
        if len(shape) == 2:
            values = rng.standard_normal(shape, dtype=np.float32)
            if name != "embed":
                values *= np.float32(1.0 / math.sqrt(shape[1]))
            bits = values.view(np.uint32)
            yield name, ((bits + 0x7fff + ((bits >> 16) & 1)) >> 16).astype(np.uint16)
        elif name.endswith(".sink"):
            yield name, rng.normal(1.0, 1.0, shape).astype(np.float32)
        elif name.endswith(".dt_bias"):
            steps = np.exp(rng.uniform(math.log(0.001), math.log(0.3), shape))
            yield name, (steps + np.log(-np.expm1(-steps))).astype(np.float32)      # softplus of it is the step
        elif name.endswith(".A_log"):
            yield name, np.log(rng.uniform(1.0, 16.0, shape)).astype(np.float32)
        elif name.endswith(".conv.b"):
            yield name, rng.normal(0.0, 0.2, shape).astype(np.float32)
        else:
            yield name, rng.uniform(0.5, 1.5, shape).astype(np.float32)


def tufirax_active_parameters(config: dict) -> int:
    """Matrix elements one token's pass multiplies with (a shared layer counts every time it runs; the head included)."""
    shapes, total = tufirax_shapes(config), config["vocab"] * config["width"]
    for i, layer in enumerate(config["layers"]):
        while "weights_of" in config["layers"][i]:
            i = config["layers"][i]["weights_of"]
        total += sum(s[0] * s[1] for n, s in shapes.items() if n.startswith(f"l{i}.") and len(s) == 2 and not n.endswith(".conv"))
    return total


def model_weight_bytes(name: str, config: dict | None = None) -> int:
    """Native GGUF bytes one decode pass streams: every matrix once, the tied head included."""
    config = config or model_config(name)
    types = tensor_types(name, config)
    shapes = matrix_shapes(config)
    total = 0
    for l in range(config["layers"]):
        for t, (k, n) in shapes.items():
            total += weight_bytes(types[f"blk.{l}.{t}.weight"], k, n)
        total += 4 * (4 * config["hidden"] + (2 * config["head_dim"] if config["uses_qk_norm"] else 0))
    head = types.get("output.weight", types["token_embd.weight"])
    total += weight_bytes(head, config["hidden"], config["vocab"]) + 4 * config["hidden"]
    return total
