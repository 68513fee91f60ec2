"""CPU checks of the layered models' host side: the plain implementation against independent arithmetic, the registry
and its errors, the reader of model folders up to the point where a device is needed."""
import ctypes as C
import json
import struct

import numpy as np
import pytest

from oracle import zasevik as z
from guffin_b200 import lib, model as gm, synthetic as syn


def tiny(**changes):
    config = syn.zasevik_config(40, 2, 3, 8, 12, 20, 50, [syn.dense_mlp(24), syn.expert_mlp(16, 5, 2, 0.8, 24, 1.1)])
    return dict(config, **changes)


def create(config, precision=0):
    L, handle = lib.load(), C.c_void_p()
    status = L.gf_model_create_described(json.dumps(config).encode() if isinstance(config, dict) else config, 64, 2, precision, C.byref(handle))
    text = L.gf_last_error().decode()
    if status == lib.GF_OK:
        L.gf_model_destroy(handle.value)
    return status, text


def test_registry_names_every_family():
    assert {"Gemma2", "Gemma3", "Zasevik"} <= set(gm.architectures())


@pytest.mark.parametrize("change, complaint", [
    (dict(architecture="Nobody"), "no architecture named 'Nobody'"),
    (dict(width=None), "width has the wrong type"),
    (dict(norm={}), "norm.eps is missing"),
    (dict(layers=[]), "layers is empty"),
    (dict(vocab=2.5), "vocab is out of range"),
])
def test_configuration_errors_name_the_value(change, complaint):
    status, text = create(tiny(**change))
    assert status == lib.GF_ERR_INVALID and complaint in text


def test_unknown_layer_kinds_are_refused():
    config = tiny()
    config["layers"][1]["type"] = "linear"
    status, text = create(config)
    assert status == lib.GF_ERR_INVALID and "layers[1].type" in text
    config = tiny()
    config["layers"][0]["mlp"]["kind"] = "sparse"
    status, text = create(config)
    assert status == lib.GF_ERR_INVALID and "layers[0].mlp.kind" in text
    config = tiny()
    config["layers"][1]["mlp"]["router"]["top"] = 6
    assert create(config)[0] == lib.GF_ERR_INVALID


def test_malformed_json_is_refused_at_its_place():
    for text in (b"", b"{", b'{"architecture": "Zasevik",}', b'{"architecture": 3}', b"[1, 2]", b'{"a": tru}'):
        assert create(text)[0] == lib.GF_ERR_INVALID


def test_escapes_and_nesting_in_json():
    status, text = create(b'{"x": {"y": [1, -2.5e3, "a\\u0041\\n", null, true]}, "architecture": "No\\u0062ody"}')
    assert status == lib.GF_ERR_INVALID and "'Nobody'" in text


def test_the_quantised_families_have_no_32_bit_form():
    config = dict(syn.model_config("tiny-target"), architecture="Gemma3")
    status, text = create(config, precision=1)
    assert status == lib.GF_ERR_INVALID and "quantised" in text


def test_a_folder_without_files_is_refused(tmp_path):
    L, handle = lib.load(), C.c_void_p()
    assert L.gf_model_open(str(tmp_path).encode(), 64, 2, 0, C.byref(handle)) == lib.GF_ERR_INVALID
    assert b"config.json" in L.gf_last_error()


# ---- the plain implementation, mechanism by mechanism

def test_norms():
    x = np.array([[3.0, -4.0]])
    want = x / np.sqrt(12.5 + 0.5)
    assert np.allclose(z.rms_norm(x, np.array([2.0, 1.0]), 0.5), want * [2.0, 1.0])
    assert np.allclose(z.centred_rms_norm(x, np.array([1.0, 0.0]), 0.5), want * [2.0, 1.0])


def test_activations():
    assert np.allclose(z.squared_relu(np.array([-3.0, 0.5, 2.0])), [0.0, 0.25, 4.0])
    # gate above, up below their limits; and neither
    gate, up = np.array([5.0, -9.0, 0.25]), np.array([-7.0, 3.0, 0.5])
    g, u = np.array([1.5, -9.0, 0.25]), np.array([-1.5, 1.5, 0.5])
    assert np.allclose(z.clamped_gate(gate, up, 1.5), g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0))


def test_sink_takes_weight_without_a_value():
    w = z.softmax_with_sink(np.array([[0.0, np.log(3.0)]]), np.log(4.0))
    assert np.allclose(w, [[1.0 / 8.0, 3.0 / 8.0]])


def test_attention_is_causal_and_scaled():
    rng = np.random.default_rng(0)
    heads, dim, vdim, rank, T, first = 2, 3, 5, 7, 4, 6
    c, q = rng.standard_normal((first + T, rank)), rng.standard_normal((T, heads * dim))
    uk, uv, sink = rng.standard_normal((heads * dim, rank)), rng.standard_normal((heads * vdim, rank)), rng.standard_normal(heads)
    got = z.latent_attention(q, c, first, heads, uk, uv, sink, 0.3)
    for t in range(T):
        for h in range(heads):
            k, v = c @ uk[h * dim:(h + 1) * dim].T, c @ uv[h * vdim:(h + 1) * vdim].T
            e = np.exp([0.3 * float(q[t, h * dim:(h + 1) * dim] @ k[j]) for j in range(first + t + 1)])
            want = (e[:, None] * v[:first + t + 1]).sum(0) / (e.sum() + np.exp(sink[h]))
            assert np.allclose(got[t, h * vdim:(h + 1) * vdim], want)


def test_absorbed_queries_score_like_expanded_keys():
    """The identity the cache layout rests on: q . (W_uk c) = (W_uk^T q) . c."""
    rng = np.random.default_rng(1)
    uk, q, c = rng.standard_normal((6, 9)), rng.standard_normal(6), rng.standard_normal(9)
    assert np.isclose(q @ (uk @ c), (uk.T @ q) @ c)


def test_routing_weights_are_the_scores_and_multiply_the_input():
    rng = np.random.default_rng(2)
    spec = syn.expert_mlp(4, 3, 2, 0.7)
    w = {"m.router": rng.standard_normal((3, 6))}
    for e in range(3):
        w.update({f"m.e{e}.gate": rng.standard_normal((4, 6)), f"m.e{e}.up": rng.standard_normal((4, 6)), f"m.e{e}.down": rng.standard_normal((6, 4))})
    h = rng.standard_normal((1, 6))
    scores = 1.0 / (1.0 + np.exp(-(h @ w["m.router"].T)[0]))
    order = np.argsort(-scores)[:2]
    want = sum(z.expert(scores[e] * h, w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"], 0.7) for e in order)
    got = z.mixture(h, w, "m", spec)
    assert np.allclose(got, want)
    after = sum(scores[e] * z.expert(h, w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"], 0.7) for e in order)
    assert not np.allclose(got, after)


def test_portions_of_the_plain_implementation_agree():
    config = tiny()
    weights = {k: gm.bf16_values(v) if v.dtype == np.uint16 else v for k, v in syn.iter_zasevik_weights(config, 3)}
    tokens = np.random.default_rng(4).integers(0, 50, 23)
    whole = z.Reference(config, weights).extend(tokens)
    cut = z.Reference(config, weights)
    parts = np.concatenate([cut.extend(tokens[a:b]) for a, b in ((0, 1), (1, 3), (3, 17), (17, 23))])
    assert np.allclose(whole, parts)


def test_shapes_cover_the_registry(tmp_path):
    """Names and shapes of the synthetic weights are those the registry lists: a file with one tensor too many, too few
    or of another shape is refused when a device is there; without one the folder is read up to the plan's creation."""
    config = tiny()
    header, blob = {}, b""
    for name, value in syn.iter_zasevik_weights(config, 5):
        data = (value if value.dtype == np.uint16 else gm.bf16_bits(value)).tobytes()
        header[name] = dict(dtype="BF16", shape=list(value.shape), data_offsets=[len(blob), len(blob) + len(data)])
        blob += data
    text = json.dumps(header).encode()
    (tmp_path / "config.json").write_text(json.dumps(config))
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + blob)
    L, handle = lib.load(), C.c_void_p()
    status = L.gf_model_open(str(tmp_path).encode(), 64, 2, 0, C.byref(handle))
    assert status in (lib.GF_OK, lib.GF_ERR_UNAVAILABLE), L.gf_last_error()
    if status == lib.GF_OK:
        L.gf_model_destroy(handle.value)
