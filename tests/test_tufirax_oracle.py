"""CPU checks of the Tufirax design's host side: the plain implementation against independent arithmetic, the
registry's reading of its configurations and its errors."""
import ctypes as C
import json

import numpy as np
import pytest

from guffin_b200 import lib, model as gm, synthetic as syn
from oracle import tufirax as o


def tiny(**changes):
    config = syn.tufirax_config(20, 30, [syn.tufirax_attention(4, 2, 6, rot_dims=4, softcap=8.0, ff=12), syn.tufirax_state_space(4, 3, 5, 2, 3, 2),
                                         syn.tufirax_attention(4, 2, 6, rot_dims=4, softcap=8.0, ff=12, weights_of=0),
                                         syn.tufirax_state_space(4, 3, 5, 2, 3, 2, weights_of=1)])
    return dict(config, **changes)


def values(config, seed):
    return {k: gm.bf16_values(v) if v.dtype == np.uint16 else v for k, v in syn.iter_tufirax_weights(config, seed)}


def create(config):
    L, handle = lib.load(), C.c_void_p()
    status = L.gf_model_create_described(json.dumps(config).encode(), 64, 2, 0, C.byref(handle))
    text = L.gf_last_error().decode()
    if status == lib.GF_OK:
        L.gf_model_destroy(handle.value)
    return status, text


def changed(layer, **changes):
    """The tiny configuration with changes to a layer: mixer.x or plain keys."""
    config = json.loads(json.dumps(tiny()))
    for key, value in changes.items():
        into = config["layers"][layer]
        *path, last = key.split("__")
        for part in path:
            into = into[part]
        if value is None:
            del into[last]
        else:
            into[last] = value
    return config


def test_the_registry_reads_the_design():
    assert "Tufirax" in gm.architectures()
    assert create(tiny())[0] in (lib.GF_OK, lib.GF_ERR_UNAVAILABLE)


@pytest.mark.parametrize("config, complaint", [
    (tiny(norm={}), "norm.eps is missing"),
    (changed(0, type="windowed"), "layers[0].type names the unknown mixer 'windowed'"),
    (changed(0, mixer__kv_heads=3), "layers[0].mixer.kv_heads does not divide"),
    (changed(0, mixer__vdim=5), "layers[0].mixer.vdim differs"),
    (changed(0, mixer__rot__dims=8), "layers[0].mixer.rot.dims"),
    (changed(0, mixer__rot__dims=3), "layers[0].mixer.rot.dims"),
    (changed(0, mixer__rot=None), "layers[0].mixer.rot is missing"),
    (changed(0, mixer__softcap=0.0), "layers[0].mixer.softcap"),
    (changed(0, mlp__kind="moe"), "layers[0].mlp.kind"),
    (changed(1, mixer__groups=3), "layers[1].mixer.groups does not divide"),
    (changed(1, mixer__norm_groups=5), "layers[1].mixer.norm_groups does not divide"),
    (changed(1, mixer__state=0), "layers[1].mixer.state is out of range"),
    (changed(2, weights_of=1), "layers[2].weights_of names a layer of another shape"),
    (changed(2, weights_of=4), "layers[2].weights_of is out of range"),
    (changed(0, weights_of=2), "weights_of leads round in a circle"),
])
def test_configuration_errors_name_the_value(config, complaint):
    status, text = create(config)
    assert status == lib.GF_ERR_INVALID and complaint in text


def test_norm_in_parts():
    x = np.array([[3.0, -4.0, 1.0, 1.0]])
    want = np.concatenate([x[:, :2] / np.sqrt(12.5 + 0.5), x[:, 2:] / np.sqrt(1.5)], axis=1) * [1.0, 2.0, 3.0, 4.0]
    assert np.allclose(o.rms_norm_in_parts(x, np.array([1.0, 2.0, 3.0, 4.0]), 2, 0.5), want)
    assert np.allclose(o.rms_norm_in_parts(x, 1.0, 1, 0.5), o.rms_norm(x, 1.0, 0.5))


def test_rotation_turns_pairs_half_apart():
    x = np.random.default_rng(0).standard_normal((3, 2, 7))
    got = o.rotate_halves(x, [0, 5, 900], 50.0, 4)
    assert np.allclose(got[0], x[0]) and np.allclose(got[..., 4:], x[..., 4:])
    for t, position in ((1, 5), (2, 900)):
        for i, f in ((0, 1.0), (1, 50.0 ** -0.5)):
            turned = (x[t, :, i] + 1j * x[t, :, i + 2]) * np.exp(1j * position * f)
            assert np.allclose(got[t, :, i], turned.real) and np.allclose(got[t, :, i + 2], turned.imag)


def test_rotated_scores_depend_on_the_distance_alone():
    q, k = np.random.default_rng(1).standard_normal((2, 1, 1, 8))
    score = lambda a, b: float((o.rotate_halves(q, [a], 100.0, 6) * o.rotate_halves(k, [b], 100.0, 6)).sum())
    assert np.isclose(score(40, 7), score(333, 300))


def test_attention_caps_scores_and_adds_the_sink():
    rng = np.random.default_rng(2)
    heads, groups, dim, T, first = 4, 2, 3, 3, 5
    q, k, v = rng.standard_normal((T, heads, dim)), rng.standard_normal((first + T, groups, dim)), rng.standard_normal((first + T, groups, dim))
    sink = rng.standard_normal(heads)
    got = o.grouped_attention(q, k, v, first, 2.0, 1.5, sink)
    for t in range(T):
        for h in range(heads):
            e = [np.exp(1.5 * np.tanh(2.0 * float(q[t, h] @ k[j, h // 2]) / 1.5)) for j in range(first + t + 1)]
            want = sum(a * v[j, h // 2] for j, a in enumerate(e)) / (sum(e) + np.exp(sink[h]))
            assert np.allclose(got[t, h], want)


def test_convolution_looks_back_and_no_further():
    rng = np.random.default_rng(3)
    x, taps, bias = rng.standard_normal((6, 2)), rng.standard_normal((2, 4)), rng.standard_normal(2)
    got = o.causal_convolution(x, np.zeros((3, 2)), taps, bias)
    for t in range(6):
        want = bias + sum(taps[:, 3 - back] * x[t - back] for back in range(4) if back <= t)
        assert np.allclose(got[t], want)
    assert np.allclose(o.causal_convolution(x[3:], x[:3], taps, bias), got[3:])


def test_the_state_is_the_decayed_sum_of_outer_products():
    rng = np.random.default_rng(4)
    heads, N, vdim, T = 2, 3, 4, 5
    x, b, c = rng.standard_normal((T, heads, vdim)), rng.standard_normal((T, heads, N)), rng.standard_normal((T, heads, N))
    dt, a_log, skip = rng.uniform(0.1, 1.0, (T, heads)), rng.standard_normal(heads), rng.standard_normal(heads)
    state = np.zeros((heads, N, vdim))
    for t in range(T):
        state, y = o.state_space_step(state, x[t], b[t], c[t], dt[t], a_log, skip)
        for h in range(heads):
            want = sum(np.exp(-np.exp(a_log[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (c[t, h] @ b[s, h]) * x[s, h] for s in range(t + 1)) + skip[h] * x[t, h]
            assert np.allclose(y[h], want)


def test_activations():
    z = np.linspace(-6.0, 6.0, 25)
    assert np.allclose(o.silu(z), z / (1.0 + np.exp(-z))) and np.allclose(o.softplus(z), np.log(1.0 + np.exp(z)))
    assert np.allclose(o.softplus(np.array([-800.0, 800.0])), [0.0, 800.0])
    want = 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))
    assert np.allclose(o.gelu_tanh(z), want)


def test_portions_of_the_plain_implementation_agree():
    config = tiny()
    weights = values(config, 3)
    tokens = np.random.default_rng(4).integers(0, 30, 23)
    whole = o.Reference(config, weights).extend(tokens)
    cut = o.Reference(config, weights)
    parts = np.concatenate([cut.extend(tokens[a:b]) for a, b in ((0, 1), (1, 3), (3, 17), (17, 23))])
    assert np.allclose(whole, parts)


def test_layers_that_share_tensors_keep_caches_of_their_own():
    config = tiny()
    weights = values(config, 5)
    copies = {k.replace("l0.", "l2.").replace("l1.", "l3."): v for k, v in weights.items()}
    apart = dict(config, layers=[{k: v for k, v in layer.items() if k != "weights_of"} for layer in config["layers"]])
    tokens = np.arange(12)
    shared = o.Reference(config, weights)
    assert np.allclose(shared.extend(tokens), o.Reference(apart, {**weights, **copies}).extend(tokens))
    assert not np.allclose(shared.keys[0], shared.keys[2]) and not np.allclose(shared.states[1], shared.states[3])
