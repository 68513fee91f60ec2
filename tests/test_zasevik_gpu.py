"""Layered models on the GPU against the plain implementation (oracle/zasevik.py): every operator alone, then whole
models of several shapes in both precisions, cut and batched in every way the plan offers."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from guffin_b200 import synthetic as syn
from oracle import zasevik as z
from tests.layered import greedy_reference, limits_of, rel_l2, row_errors, tokens_for, within, write_folder

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
SERVING, F32 = 0, 1


@pytest.fixture(scope="module")
def gm(gf):
    from guffin_b200 import model
    return model


def plain(config, weights, tokens, precision):
    return limits_of(z.Reference, z.bf16, config, weights, tokens, precision)


# ------------------------------------------------------------------------------------------- operators

def packed(gf, gm, rng, k, n):
    bits = gm.bf16_bits(rng.standard_normal((n, k)))
    src, dst = gf.DeviceBuffer.from_numpy(bits), gf.DeviceBuffer(gf.load().gf_dense_packed_bytes(k, n))
    gf.check(gf.load().gf_dense_pack(src.ptr, k, n, dst.ptr, None))
    gf.check(gf.load().gf_stream_synchronize(None))
    return dst, gm.bf16_values(bits).astype(np.float64)


@pytest.mark.parametrize("k,n", [(7, 5), (33, 130), (96, 64), (200, 257), (1030, 24), (6400, 40)])
def test_row_products(gf, gm, k, n):
    rng = np.random.default_rng(k)
    weight, w = packed(gf, gm, rng, k, n)
    x = rng.standard_normal((11, k)).astype(np.float32)
    xd = gf.DeviceBuffer.from_numpy(x)
    results = {}
    for rows in (1, 2, 3, 4, 5, 6, 7, 8, 11):
        y = gf.DeviceBuffer(rows * n * 4)
        gf.check(gf.load().gf_dense_matmul(weight.ptr, xd.ptr, y.ptr, rows, k, n, None))
        results[rows] = y.download(np.float32).reshape(rows, n)
        assert rel_l2(results[rows], x[:rows] @ w.T) < 2e-6
    for rows in results:                       # a row's sum does not depend on the rows beside it
        assert np.array_equal(results[rows][0], results[1][0])


@pytest.mark.parametrize("k,n", [(7, 5), (72, 130), (200, 257), (1030, 24)])
@pytest.mark.parametrize("rows", [1, 16, 17, 130, 300])
def test_chunk_products(gf, gm, k, n, rows):
    rng = np.random.default_rng(rows)
    weight, w = packed(gf, gm, rng, k, n)
    x = rng.standard_normal((rows, k)).astype(np.float32)
    xd, y = gf.DeviceBuffer.from_numpy(x), gf.DeviceBuffer(rows * n * 4)
    for precision, operand, bound in ((SERVING, gm.bf16_values(gm.bf16_bits(x)), 2e-6), (F32, x, 2e-6)):
        ws = gf.DeviceBuffer(gf.load().gf_dense_chunk_workspace_bytes(rows, k, precision))
        ws.zero()
        gf.check(gf.load().gf_dense_chunk_matmul(weight.ptr, xd.ptr, y.ptr, rows, k, n, precision, ws.ptr, None))
        assert rel_l2(y.download(np.float32).reshape(rows, n), operand.astype(np.float64) @ w.T) < bound


def run_attention(gf, q, cache, first, rows, sink, parts, precision, ring_rows):
    """q [rows, heads, rank] scaled, cache [first + rows, rank]: device result [rows, heads, rank]."""
    heads, rank = q.shape[1:]
    dtype, wide = (np.float32 if precision == F32 else np.float16), (rank + 15) // 16 * 16
    pad = lambda a: np.pad(a, [(0, 0)] * (a.ndim - 1) + [(0, wide - rank)]).astype(dtype)
    ring = np.full((ring_rows, wide), 7.0, dtype)
    for position in range(max(0, first - ring_rows), first):
        ring[position % ring_rows] = pad(cache[position:position + 1])[0]
    buffers = [gf.DeviceBuffer.from_numpy(a) for a in (pad(q).reshape(rows * heads, wide), ring, pad(cache[first:]), np.array([first, 0, 0, 0], np.uint32))]
    sink_dev = gf.DeviceBuffer.from_numpy(np.asarray(sink, np.float32)) if sink is not None else None
    out = gf.DeviceBuffer(rows * heads * wide * 4)
    ws = gf.DeviceBuffer(gf.load().gf_latent_attention_workspace_bytes(rows, heads, rank, parts))
    gf.check(gf.load().gf_latent_attention(buffers[0].ptr, buffers[1].ptr, buffers[2].ptr, buffers[3].ptr, sink_dev.ptr if sink_dev else None, out.ptr,
                                           rows, heads, rank, ring_rows, parts, precision, ws.ptr, None))
    return out.download(np.float32).reshape(rows, heads, wide)[:, :, :rank]


def plain_attention(q, cache, first, sink):
    rows, heads, rank = q.shape
    eye, out = np.eye(rank), np.empty(q.shape)
    for h in range(heads):
        out[:, h] = z.latent_attention(q[:, h].astype(np.float64), cache.astype(np.float64), first, 1, eye, eye,
                                       [-np.inf if sink is None else sink[h]], 1.0)
    return out


@pytest.mark.parametrize("precision,bound", [(SERVING, 2e-3), (F32, 2e-6)])
@pytest.mark.parametrize("rank,heads,rows,first,parts", [
    (20, 3, 1, 0, 1), (20, 3, 5, 63, 2), (48, 1, 8, 64, 3), (130, 16, 1, 129, 4), (256, 7, 3, 200, 128), (512, 5, 17, 65, 1), (272, 16, 2, 190, 5), (600, 2, 2, 70, 2)])
def test_latent_attention(gf, precision, bound, rank, heads, rows, first, parts):
    rng = np.random.default_rng(rank + rows)
    dtype = np.float32 if precision == F32 else np.float16
    q = (rng.standard_normal((rows, heads, rank)) * 2.0 / np.sqrt(rank)).astype(dtype)
    cache = rng.standard_normal((first + rows, rank)).astype(dtype)
    for sink in (None, rng.normal(1.0, 1.0, heads).astype(np.float32)):
        got = run_attention(gf, q, cache, first, rows, sink, parts, precision, 256)
        assert rel_l2(got, plain_attention(q, cache, first, sink)) < bound


@pytest.mark.parametrize("precision", [SERVING, F32])
def test_attention_finds_one_key(gf, precision):
    """One key stands out: at the first position, at tile borders, inside the pass's own rows, on the row itself."""
    rng = np.random.default_rng(9)
    rank, heads, rows, first = 32, 4, 6, 190
    dtype = np.float32 if precision == F32 else np.float16
    for place in (0, 1, 63, 64, 127, 128, 189, 190, 193, 195):
        cache = (rng.standard_normal((first + rows, rank)) * 0.1).astype(dtype)
        q = rng.standard_normal((rows, heads, rank)).astype(dtype)
        direction = q[rows - 1, 2].astype(np.float64)
        cache[place] = (direction * 30.0 / (direction @ direction)).astype(dtype)
        got = run_attention(gf, q, cache, first, rows, np.zeros(heads), 3, precision, 256)
        want = plain_attention(q, cache, first, np.zeros(heads))
        assert rel_l2(got, want) < 3e-3 and rel_l2(got[rows - 1, 2], cache[place].astype(np.float64)) < 1e-2
        if place > first:                       # the row just before it must not see it
            assert rel_l2(got[place - first - 1, 2], want[place - first - 1, 2]) < 3e-3


def test_routing(gf):
    rng = np.random.default_rng(5)
    for rows, experts, top in ((1, 1, 1), (7, 5, 2), (33, 64, 6), (3, 100, 9)):
        logits = rng.standard_normal((rows, experts)).astype(np.float32)
        logits[0] = np.where(np.arange(experts) % 2, 1.0, 1.0)                       # ties go to the lower index
        src, ids, scores = gf.DeviceBuffer.from_numpy(logits), gf.DeviceBuffer(rows * top * 4), gf.DeviceBuffer(rows * top * 4)
        gf.check(gf.load().gf_route(src.ptr, rows, experts, top, ids.ptr, scores.ptr, None))
        want, weights = z.route(logits.astype(np.float64), np.eye(experts), top)
        assert np.array_equal(ids.download(np.uint32).reshape(rows, top), want)
        assert np.allclose(scores.download(np.float32).reshape(rows, top), weights, rtol=1e-6)


# ------------------------------------------------------------------------------------------- whole models

def layer(heads, dim, vdim, rank, scale, mlp):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale), mlp=mlp)


def described(width, vocab, eps, scale, layers):
    return dict(architecture="Zasevik", embedding=dict(scale=scale), norm=dict(eps=eps), vocab=vocab, width=width, layers=layers)


CONFIGS = {
    "dense, ragged sizes": described(40, 53, 1e-5, 5.0, [layer(3, 8, 12, 20, 0.5, syn.dense_mlp(24)), layer(3, 8, 12, 20, 0.5, syn.dense_mlp(24))]),
    "attention alone": described(50, 61, 1e-3, 1.0, [layer(2, 10, 6, 36, 1.3, None), layer(2, 10, 6, 36, 1.3, None)]),
    "sharp attention": described(64, 96, 1e-6, 2.0, [layer(4, 16, 16, 48, 2.5, None), layer(1, 64, 32, 16, 1.5, syn.dense_mlp(40))]),
    "experts": described(72, 80, 1e-6, 8.0, [layer(5, 24, 16, 40, 0.3, syn.expert_mlp(20, 7, 3, 0.6, 36, 0.9)), layer(5, 24, 16, 40, 0.3, syn.expert_mlp(33, 4, 1, 2.5))]),
    "every layer its own sizes": described(96, 128, 1e-6, 3.0, [
        layer(2, 40, 24, 30, 0.2, syn.expert_mlp(48, 6, 2, 1.0, 16, 0.5)), layer(6, 8, 20, 112, 0.4, None), layer(3, 20, 40, 64, 0.25, syn.dense_mlp(100)),
        layer(1, 16, 8, 144, 0.3, syn.expert_mlp(8, 9, 9, 0.7))]),
    "wide latents": described(128, 160, 1e-6, 11.0, [layer(4, 32, 64, 320, 0.18, syn.dense_mlp(200)), layer(4, 64, 32, 512, 0.12, syn.expert_mlp(64, 8, 2, 1.2, 40, 1.4))]),
}


SEEDS = {"every layer its own sizes": 6, "wide latents": 7}      # the smallest routing margin is far above rounding


def make(gm, name, seed=None):
    """Weights as the product takes them and as the plain implementation does.  In models with experts every token's
    embedding ranks the experts in a random order, by levels far apart in as many places as there are experts, and the
    routers read these places: rounding then chooses the same experts, and a wrong choice shows."""
    seed = seed or SEEDS.get(name, 4)
    config, rng = CONFIGS[name], np.random.default_rng(seed)
    values = {k: gm.bf16_values(v) if v.dtype == np.uint16 else v for k, v in syn.iter_zasevik_weights(config, seed)}
    experts = [l["mlp"]["router"]["experts"] if l["mlp"] and l["mlp"]["kind"] == "moe" else 0 for l in config["layers"]]
    most = max(experts)
    if most:
        levels = np.linspace(-4.0, 4.0, most) / config["embedding"]["scale"] * np.sqrt(config["width"])
        for token in range(config["vocab"]):
            values["embed"][token, :most] = rng.permutation(levels)
        for i, count in enumerate(experts):
            if count:
                values[f"l{i}.mlp.router"] = np.eye(count, config["width"]) * 1.5 + 0.02 * rng.standard_normal((count, config["width"]))
        values["final.norm"][:most] = -0.95              # these places say little about the next token
    bits = {k: gm.bf16_bits(v) for k, v in values.items()}
    return config, bits, {k: gm.bf16_values(v) for k, v in bits.items()}


PRECISIONS = ["float32", "bfloat16"]


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("precision", PRECISIONS)
def test_whole_prompts_and_rows(gm, name, precision):
    """A prompt as one portion (chunks on the tensor cores, or 32-bit ones) and as row passes; latents of every layer too."""
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 150)
    want, limits = plain(config, weights, tokens, precision)
    ref, rounded = z.Reference(config, weights), z.Reference(config, weights, cast=z.bf16)
    ref.extend(tokens), rounded.extend(tokens)
    plan = gm.Model.described(config, bits, 200, 8, precision)
    for chunks in (True, False):
        plan.reset()
        plan.use_tensor_prefill(chunks)
        got = plan.extend(tokens, range(150))
        assert within(got, want, limits), chunks
        for l in range(len(config["layers"])):
            latents = plan.read_latents(l, 0, 150)
            assert rel_l2(latents, ref.latents[l]) < (2e-6 if precision == "float32" else 2.0 * rel_l2(rounded.latents[l], ref.latents[l])), l
    assert plan.status() == 0 and plan.position == 150


@pytest.mark.parametrize("name", ["dense, ragged sizes", "experts", "every layer its own sizes", "wide latents"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_portions_of_every_size(gm, name, precision):
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 200, 1)
    want, limits = plain(config, weights, tokens, precision)
    plan = gm.Model.described(config, bits, 200, 8, precision)
    for cuts in ([2] * 100, [1, 16, 17, 2, 64, 3, 65, 2, 30], [199, 1], [33, 100, 67], [9, 8, 183]):
        plan.reset()
        at, rows = 0, []
        for size in cuts:
            rows.append(plan.extend(tokens[at:at + size], range(size)))
            at += size
        assert at == 200 and within(np.concatenate(rows), want, limits), cuts


@pytest.mark.parametrize("name", ["sharp attention", "experts"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_prompts_longer_than_a_chunk(gm, name, precision):
    """The second chunk of a long prompt sees the first one's cache rows; only some logits are wanted."""
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 1100, 5)
    want, limits = plain(config, weights, tokens, precision)
    places = [0, 1, 511, 1022, 1023, 1024, 1025, 1060, 1099]
    plan = gm.Model.described(config, bits, 1100, 8, precision)
    assert within(plan.extend(tokens, places), want[places], limits[places])
    plan.reset()
    plan.extend(tokens[:1090])
    assert within(plan.extend(tokens[1090:], [0, 9]), want[[1090, 1099]], limits[[1090, 1099]])


@pytest.mark.parametrize("precision", PRECISIONS)
def test_decoding_behind_a_prompt(gm, precision):
    """Token by token for longer than the prompt, through the captured passes, up to the last position of the context."""
    config, bits, weights = make(gm, "every layer its own sizes")
    tokens = tokens_for(config, 300, 2)
    want, limits = plain(config, weights, tokens, precision)
    plan = gm.Model.described(config, bits, 300, 4, precision)
    plan.prefill(tokens[:70])
    assert within(plan.logits(plan.prefill_logits_row)[None], want[69:70], limits[69:70])
    got = []
    for t in range(70, 300):
        plan.forward(tokens[t:t + 1])
        plan.publish(1)
        got.append(plan.logits(0))
    assert within(np.stack(got), want[70:], limits[70:])
    with pytest.raises(Exception, match="exceeds the bound context"):
        plan.extend(tokens[:1])
    # several rows per pass, unpublished rows thrown away and written again
    plan.reset()
    plan.prefill(tokens[:50])
    plan.forward(tokens[:3])
    plan.forward(tokens[50:54])
    plan.publish(2)
    plan.forward(tokens[52:56])
    assert within(np.stack([plan.logits(r) for r in range(4)]), want[52:56], limits[52:56])


@pytest.mark.parametrize("precision", PRECISIONS)
def test_first_tokens_and_reset(gm, precision):
    """One token alone: its own key and the sink share the softmax.  A plan that is reset repeats itself bit for bit."""
    config, bits, weights = make(gm, "sharp attention")
    plan = gm.Model.described(config, bits, 64, 8, precision)
    for token in (0, 1, config["vocab"] - 1):
        plan.reset()
        got = plan.extend([token], [0])
        assert row_errors(got, z.Reference(config, weights).extend([token])).max() < (2e-5 if precision == "float32" else 4e-3)
    tokens = tokens_for(config, 40, 3)
    plan.reset()
    first = plan.extend(tokens, range(40))
    plan.extend(tokens[:20])
    plan.reset()
    assert np.array_equal(first, plan.extend(tokens, range(40)))
    with pytest.raises(Exception, match="outside the vocabulary"):
        plan.extend([config["vocab"]], [0])
    with pytest.raises(Exception, match="wanted places"):
        plan.extend([1, 2], [1, 0])


@pytest.mark.parametrize("precision", PRECISIONS)
def test_a_key_far_away(gm, precision):
    """Tokens far apart that ask for one another: large embeddings along one direction and a sharp score make the far key
    win over hundreds of others, in prompts, in portions and in decoding."""
    config = described(48, 40, 1e-6, 4.0, [layer(2, 16, 16, 24, 4.0, None)] * 2)
    weights = {k: v if v.dtype == np.uint16 else gm.bf16_bits(v) for k, v in syn.iter_zasevik_weights(config, 6)}
    values = {k: gm.bf16_values(v) for k, v in weights.items()}
    tokens = tokens_for(config, 420, 4) % 38
    tokens[[0, 64, 200]], tokens[[150, 320, 419]] = 38, 39                          # rare tokens, met again far behind
    want, limits = plain(config, values, tokens, precision)
    other = tokens.copy()
    other[0] = 5
    moved = row_errors(z.Reference(config, values).extend(other), want)
    assert moved[319] > 1e-4                                                       # the far token shows in the logits
    plan = gm.Model.described(config, weights, 420, 8, precision)
    assert within(plan.extend(tokens, range(420)), want, limits)
    plan.reset()
    plan.extend(tokens[:400])
    got = [plan.extend(tokens[t:t + 1], [0])[0] for t in range(400, 420)]
    assert within(np.stack(got), want[400:], limits[400:])


@pytest.mark.parametrize("precision", PRECISIONS)
def test_streams_equal_conversations_alone(gm, precision):
    """Unequal conversations decoded together, in groups smaller than their number; a slot given back and used again."""
    config, bits, weights = make(gm, "experts")
    plan = gm.Model.described(config, bits, 160, 4, precision)
    streams = gm.Streams(plan, 6)
    prompts = [tokens_for(config, n, n) for n in (1, 30, 64, 65, 7, 130)]
    feeds = tokens_for(config, 6 * 12, 9).reshape(12, 6)
    for s, prompt in enumerate(prompts):
        streams.prefill(s, prompt)
    assert np.array_equal(streams.greedy(), [int(np.argmax(streams.logits(s))) for s in range(6)])
    got = {s: [streams.logits(s)] for s in range(6)}
    for step in feeds:
        streams.decode(step)
        for s in range(6):
            got[s].append(streams.logits(s))
    for s, prompt in enumerate(prompts):
        want, limits = plain(config, weights, np.concatenate([prompt, feeds[:, s]]), precision)
        assert within(np.stack(got[s]), want[prompt.size - 1:], limits[prompt.size - 1:]), s
    assert plan.position == 0                                                       # the plan's own cache was left alone
    streams.release(5)
    short = tokens_for(config, 21, 77)
    again = streams.extend(5, short, range(21))
    assert within(again, *plain(config, weights, short, precision))
    assert [streams.position(s) for s in range(6)] == [p.size + 12 for p in prompts[:5]] + [21]
    streams.decode(feeds[0])
    want, limits = plain(config, weights, np.concatenate([prompts[2], feeds[:, 2], feeds[0, 2:3]]), precision)
    assert within(streams.logits(2)[None], want[-1:], limits[-1:])


@pytest.mark.parametrize("name", ["sharp attention", "every layer its own sizes"])
def test_greedy_generation(gm, name):
    """The generation engine, the batch, the engine with a drafter, and the plain implementation choose the same tokens."""
    from guffin_b200 import engine as ge
    config, bits, weights = make(gm, name)
    plan = gm.Model.described(config, bits, 256, 4, "float32")
    prompts = [tokens_for(config, n, n) for n in (40, 3, 90)]
    wanted = [greedy_reference(z.Reference, config, weights, p, 48) for p in prompts]
    assert all(margin > 1e-3 for _, margin in wanted) and (name != "sharp attention" or len(set(wanted[0][0])) > 10)
    options = ge.sampler_options(0.0)
    engine = ge.H1(plan, None, ge.H1Options(options, 0, 0, 0.0, 0, 0))
    for prompt, (want, _) in zip(prompts, wanted):
        engine.prefill(prompt)
        assert engine.generate(48).tolist() == want
    batch = ge.Batch(plan, prompts, options)
    assert batch.generate(48).tolist() == [want for want, _ in wanted]
    draft = gm.Model.described(config, {k: (gm.bf16_bits(gm.bf16_values(v) * 0.5) if k == "l1.mix.o" else v) for k, v in bits.items()}, 256, 2)
    speculative = ge.H1(plan, draft, ge.H1Options(options, 1, 0, 0.0, 0, 0))
    speculative.prefill(prompts[0])
    assert speculative.generate(48).tolist() == wanted[0][0]
    assert speculative.stats().cycles > 0


def test_seeded_sampling_in_a_batch(gm):
    """A stream's sampled tokens are those of the same conversation generated alone with the same seed."""
    from guffin_b200 import engine as ge
    config, bits, _ = make(gm, "experts")
    plan = gm.Model.described(config, bits, 128, 4, "float32")
    prompts = [tokens_for(config, n, n) for n in (11, 40)]
    options = [ge.sampler_options(0.9, 20, seed=s, repetition_penalty=1.1) for s in (1, 2)]
    rows = ge.Batch(plan, prompts, options).generate(24)
    for prompt, o, row in zip(prompts, options, rows):
        engine = ge.H1(plan, None, ge.H1Options(o, 0, 0, 0.0, 0, 0))
        engine.prefill(prompt)
        assert engine.generate(24).tolist() == row.tolist()


def test_what_a_layered_plan_does_not_offer(gm):
    config, bits, _ = make(gm, "attention alone")
    plan = gm.Model.described(config, bits, 64, 2)
    with pytest.raises(Exception, match="not offered"):
        plan.use_pass_kernel(1)
    with pytest.raises(Exception, match="not offered"):
        plan.weight_sweep(1)
    with pytest.raises(Exception, match="row passes"):
        gm.Streams(plan, 2).set_mode(1)
    with pytest.raises(Exception, match="has no tensor 'l9.norm1'"):
        gm.Model.described(config, dict(bits, **{"l9.norm1": bits["l0.norm1"]}), 64, 2)
    with pytest.raises(Exception, match="'final.norm' is not bound"):
        gm.Model.described(config, {k: v for k, v in bits.items() if k != "final.norm"}, 64, 2)
    with pytest.raises(Exception, match="should have shape"):
        gm.Model.described(config, dict(bits, **{"l0.mix.q": bits["l0.mix.o"]}), 64, 2)


# ------------------------------------------------------------------------------------------- folders and programs

@pytest.mark.parametrize("precision", PRECISIONS)
def test_trace_replay(gm, tmp_path, precision):
    config, bits, weights = make(gm, "experts")
    write_folder(tmp_path, config, bits)
    requests = {"a": tokens_for(config, 90, 1), "b": tokens_for(config, 33, 2), "c": tokens_for(config, 5, 3)}
    steps, expected, at = [], [], dict.fromkeys(requests, 0)
    for name, size, want in (("a", 50, [0, 49]), ("a", 2, []), ("b", 33, [32, 4]), ("a", 38, [1]), ("c", 5, [0, 4])):
        portion = requests[name][at[name]:at[name] + size]
        expected.append([(name, at[name] + w) for w in want])
        at[name] += size
        steps.append(dict(step=len(steps), entries=[dict(id=name, tokens=portion.tolist(), want=want)], end=[name] if at[name] == len(requests[name]) else []))
    out = tmp_path / "out"
    out.mkdir()
    done = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", precision, "--out", str(out), "--max-tokens", "128"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert done.returncode == 0, done.stderr
    assert [line for line in done.stdout.split("\n") if line.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    wanted = {name: plain(config, weights, tokens, precision) for name, tokens in requests.items()}
    for i, places in enumerate(expected):
        path = out / f"{i}.f32"
        assert path.exists() == bool(places)
        if places:
            got = np.fromfile(path, "<f4").reshape(len(places), -1)
            assert within(got, np.stack([wanted[n][0][p] for n, p in places]), np.array([wanted[n][1][p] for n, p in places]))


def test_command_line(gm, tmp_path):
    config, bits, weights = make(gm, "every layer its own sizes")
    write_folder(tmp_path, config, bits)
    prompt = tokens_for(config, 40, 40)
    want, _ = greedy_reference(z.Reference, config, weights, prompt, 10)
    text = ",".join(str(t) for t in prompt)
    run = lambda *args: subprocess.run([sys.executable, "-m", "guffin_b200", *args], cwd=ROOT, capture_output=True, text=True, timeout=300)
    one = run("generate", "--model", str(tmp_path), "--tokens", text, "--max-tokens", "10", "--dtype", "float32")
    assert one.returncode == 0 and one.stdout.split() == [str(t) for t in want], one.stderr
    two = run("generate", "--model", str(tmp_path), "--tokens", text, "--tokens", "1 2 3", "--max-tokens", "10", "--dtype", "float32")
    assert two.stdout.splitlines()[0].split() == [str(t) for t in want], two.stderr
    info = run("info", str(tmp_path))
    assert info.returncode == 0 and "latent_attention" in info.stdout and "Zasevik" in info.stdout
    assert "Zasevik" in run("models").stdout.split()
