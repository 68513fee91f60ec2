"""The Tufirax design on the GPU against the plain implementation (oracle/tufirax.py): every mixer alone and whole models
of several shapes in both precisions, cut and batched in every way the plan offers."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from guffin_b200 import synthetic as syn
from oracle import tufirax as o
from tests.layered import greedy_reference, limits_of, rel_l2, row_errors, tokens_for, within, write_folder

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PRECISIONS = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def gm(gf):
    from guffin_b200 import model
    return model


def plain(config, weights, tokens, precision):
    return limits_of(o.Reference, o.bf16, config, weights, tokens, precision)


attention, state_space = syn.tufirax_attention, syn.tufirax_state_space
CONFIGS = {
    "attention alone": syn.tufirax_config(45, 53, [attention(6, 3, 10, 0.5, 7.0, 4, 900.0), attention(6, 3, 10, 0.5, 7.0, 4, 900.0)], 1e-3),
    "one head": syn.tufirax_config(36, 50, [attention(1, 1, 24, 0.3, 3.0, 24, 77.0, ff=20), attention(1, 1, 7, 0.4, 50.0, 2, 10.0, ff=9)], 1e-5),
    "heads of their own": syn.tufirax_config(64, 80, [attention(5, 5, 20, 0.9, 4.0, 12, 5e4, ff=33), attention(12, 2, 40, 0.2, 12.0, 40, 300.0)]),
    "wide heads": syn.tufirax_config(72, 64, [attention(3, 1, 144, 0.08, 9.0, 64, 1e4, ff=40), attention(2, 2, 272, 0.06, 20.0, 16, 1e3)]),
    "states alone": syn.tufirax_config(37, 48, [state_space(4, 6, 5, 2, 2, 3), state_space(4, 6, 5, 2, 2, 3)], 1e-4),
    "states and feed-forwards": syn.tufirax_config(48, 60, [state_space(3, 20, 24, 1, 1, 1, ff=30), state_space(6, 9, 17, 3, 7, 2, ff=11), state_space(1, 5, 3, 1, 3, 5)]),
    "wide states": syn.tufirax_config(56, 72, [state_space(2, 70, 140, 2, 4, 7), state_space(8, 64, 128, 4, 4, 8), state_space(2, 33, 270, 1, 5, 6)]),
    "many heads": syn.tufirax_config(52, 66, [attention(20, 1, 12, 0.4, 8.0, 6, 500.0), state_space(70, 3, 9, 1, 11, 1), state_space(8, 64, 20, 2, 4, 2, ff=13)]),
    "shared in turn": syn.tufirax_config(60, 90, [
        state_space(4, 12, 20, 2, 4, 4), attention(4, 2, 18, 0.3, 6.0, 10, 2e3, ff=28), state_space(4, 12, 20, 2, 4, 4, weights_of=0),
        attention(4, 2, 18, 0.3, 6.0, 10, 2e3, ff=28, weights_of=1), attention(8, 1, 16, 0.25, 30.0, 16, 1e4), state_space(4, 12, 20, 2, 4, 4, weights_of=2),
        attention(8, 1, 16, 0.25, 30.0, 16, 1e4, weights_of=4)]),
}


def weights_for(gm, config, seed):
    """Weights as the product takes them and as the plain implementation does.  The sublayers' norms have small gains, so
    that rounding does not grow from layer to layer."""
    bits = {}
    for name, value in syn.iter_tufirax_weights(config, seed):
        value = gm.bf16_values(value) if value.dtype == np.uint16 else value
        bits[name] = gm.bf16_bits(value * 0.4 if name.endswith(("norm1", "norm2")) else value)
    return bits, {k: gm.bf16_values(v) for k, v in bits.items()}


def make(gm, name, seed=4):
    return (CONFIGS[name], *weights_for(gm, CONFIGS[name], seed))


# ------------------------------------------------------------------------------------------- whole models

@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("precision", PRECISIONS)
def test_whole_prompts_and_rows(gm, name, precision):
    """A prompt as one portion (chunks on the tensor cores, or 32-bit ones) and as row passes: logits, keys, values and states."""
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 150)
    want, limits = plain(config, weights, tokens, precision)
    ref, rounded = o.Reference(config, weights), o.Reference(config, weights, cast=o.bf16)
    ref.extend(tokens), rounded.extend(tokens)
    plan = gm.Model.described(config, bits, 200, 8, precision)

    def close(got, exact, coarse):
        assert rel_l2(got, exact) < (1e-5 if precision == "float32" else 2.0 * rel_l2(coarse, exact) + 1e-3), (chunks, l)
    for chunks in (True, False):
        plan.reset()
        plan.use_tensor_prefill(chunks)
        assert within(plan.extend(tokens, range(150)), want, limits), chunks
        for l, layer in enumerate(config["layers"]):
            if layer["type"] == "attention":
                k, v = plan.read_keys_values(l, 0, 150)
                close(k, ref.keys[l], rounded.keys[l])
                close(v, ref.values[l], rounded.values[l])
            else:
                close(plan.read_state(l), ref.states[l].transpose(0, 2, 1), rounded.states[l].transpose(0, 2, 1))
    assert plan.status() == 0 and plan.position == 150


@pytest.mark.parametrize("name", ["heads of their own", "states alone", "states and feed-forwards", "wide states", "many heads", "shared in turn"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_portions_of_every_size(gm, name, precision):
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 200, 1)
    want, limits = plain(config, weights, tokens, precision)
    plan = gm.Model.described(config, bits, 200, 8, precision)
    for cuts in ([2] * 100, [1, 16, 17, 2, 64, 3, 65, 2, 30], [199, 1], [33, 100, 67], [9, 8, 183], [18, 19, 1, 20, 142]):
        plan.reset()
        at, rows = 0, []
        for size in cuts:
            rows.append(plan.extend(tokens[at:at + size], range(size)))
            at += size
        assert at == 200 and within(np.concatenate(rows), want, limits), cuts


@pytest.mark.parametrize("state", [1, 4, 6, 11, 16, 30, 64, 100, 256, 400, 700, 1024])
def test_states_of_every_size(gm, state):
    """The recurrence has an instance per range of sizes; heads share their group's vectors, columns end inside a block."""
    config = syn.tufirax_config(24, 40, [state_space(6, 37, state, 2, 3, 1)])
    bits, weights = weights_for(gm, config, state)
    tokens = tokens_for(config, 61, 1)
    want = o.Reference(config, weights).extend(tokens)
    plan = gm.Model.described(config, bits, 64, 8, "float32")
    got = np.concatenate([plan.extend(tokens[:30], range(30)), plan.extend(tokens[30:35], range(5)), plan.extend(tokens[35:], range(26))])
    assert row_errors(got, want).max() < 1e-4


@pytest.mark.parametrize("name", ["attention alone", "shared in turn"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_prompts_longer_than_a_chunk(gm, name, precision):
    """The second chunk of a long prompt sees the first one's rows and state; only some logits are wanted, then none."""
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 1100, 5)
    want, limits = plain(config, weights, tokens, precision)
    places = [0, 1, 511, 1022, 1023, 1024, 1025, 1060, 1099]
    plan = gm.Model.described(config, bits, 1100, 8, precision)
    assert within(plan.extend(tokens, places), want[places], limits[places])
    plan.reset()
    plan.extend(tokens[:1090])
    assert within(plan.extend(tokens[1090:], [0, 9]), want[[1090, 1099]], limits[[1090, 1099]])


@pytest.mark.parametrize("name", ["heads of their own", "shared in turn"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_decoding_behind_a_prompt(gm, name, precision):
    """Token by token for longer than the prompt, through the captured passes, up to the last position of the context."""
    config, bits, weights = make(gm, name)
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


@pytest.mark.parametrize("name", ["states and feed-forwards", "shared in turn"])
def test_rows_thrown_away(gm, name):
    """Unpublished rows leave keys, states and the convolutions' inputs as they were; published ones can be taken back."""
    config, bits, weights = make(gm, name)
    tokens = tokens_for(config, 90, 6)
    want = o.Reference(config, weights).extend(tokens)
    plan = gm.Model.described(config, bits, 96, 4, "float32")
    logits = lambda rows: np.stack([plan.logits(r) for r in range(rows)])
    for start in (50, 3, 0):                   # behind a chunk, behind rows, at the start
        plan.reset()
        if start:
            plan.prefill(tokens[:start])
        plan.forward(tokens[:3])               # thrown away
        plan.forward(tokens[start:start + 4])
        assert row_errors(logits(4), want[start:start + 4]).max() < 1e-4
        plan.publish(2)
        plan.forward(tokens[40:44])            # thrown away
        plan.forward(tokens[start + 2:start + 6])
        plan.publish(4)
        plan.truncate(start + 3)
        plan.forward(tokens[start + 3:start + 7])
        assert row_errors(logits(4), want[start + 3:start + 7]).max() < 1e-4
    if any(layer["type"] == "mamba2" for layer in config["layers"]):
        plan.reset()
        plan.prefill(tokens[:60])
        with pytest.raises(Exception, match="no longer held"):
            plan.truncate(58)
        plan.forward(tokens[60:62])
        plan.publish(2)
        plan.truncate(60)
        plan.forward(tokens[60:64])
        assert row_errors(logits(4), want[60:64]).max() < 1e-4


@pytest.mark.parametrize("precision", PRECISIONS)
def test_first_tokens_and_reset(gm, precision):
    """One token alone: its own key and the sink share the softmax, nothing lies behind the convolution.  A plan that is
    reset repeats itself bit for bit."""
    config, bits, weights = make(gm, "shared in turn")
    plan = gm.Model.described(config, bits, 64, 8, precision)
    for token in (0, 1, config["vocab"] - 1):
        plan.reset()
        got = plan.extend([token], [0])
        assert row_errors(got, o.Reference(config, weights).extend([token])).max() < (2e-5 if precision == "float32" else 5e-3)
    tokens = tokens_for(config, 40, 3)
    plan.reset()
    first = plan.extend(tokens, range(40))
    plan.extend(tokens[:20])
    plan.reset()
    assert np.array_equal(first, plan.extend(tokens, range(40)))


def test_sinks_and_gates_take_part(gm):
    """A sink above every score, a gate that shuts its head: what the plain implementation says, and not what it says without."""
    config, bits, weights = make(gm, "heads of their own")
    weights = dict(weights)
    weights["l0.mix.sink"] = np.array([9.0, -9.0, 4.0, 3.5, -2.0], np.float32)
    weights["l1.mix.g"] = weights["l1.mix.g"] * np.where(np.arange(12) % 2, 8.0, -8.0)[:, None].astype(np.float32)
    bits = {k: gm.bf16_bits(v) for k, v in weights.items()}
    weights = {k: gm.bf16_values(v) for k, v in bits.items()}
    tokens = tokens_for(config, 80, 8)
    want = o.Reference(config, weights).extend(tokens)
    without = o.Reference(config, dict(weights, **{"l0.mix.sink": np.full(5, -60.0)})).extend(tokens)
    assert row_errors(without, want).min() > 1e-2
    plan = gm.Model.described(config, bits, 80, 8, "float32")
    for chunks in (True, False):
        plan.reset()
        plan.use_tensor_prefill(chunks)
        assert row_errors(plan.extend(tokens, range(80)), want).max() < 1e-4


def seeking_weights(gm, config, seed):
    """Keys (and values) read one half of a token's embedding, queries the other: token 39 asks for token 38, whose key
    stands out among all others by a score of about 10."""
    width, rng = config["width"], np.random.default_rng(seed)
    bits, _ = weights_for(gm, config, seed)
    half = width // 2
    embed = gm.bf16_values(bits["embed"]).copy()
    embed[39, half:] = embed[38, :half]
    bits["embed"] = gm.bf16_bits(embed)
    for l in range(len(config["layers"])):
        noise = lambda rows: 0.02 * rng.standard_normal((rows, width))
        eye = np.eye(half, width)
        bits[f"l{l}.mix.k"] = gm.bf16_bits(eye + noise(half))
        bits[f"l{l}.mix.q"] = gm.bf16_bits(np.concatenate([np.roll(eye, half, axis=1) + noise(half), rng.standard_normal((half, width)) / np.sqrt(width)]))
        for name in ("q", "k"):
            bits[f"l{l}.mix.{name}.norm"] = gm.bf16_bits(np.ones(bits[f"l{l}.mix.{name}.norm"].shape))
    return bits, {k: gm.bf16_values(v) for k, v in bits.items()}


@pytest.mark.parametrize("precision", PRECISIONS)
def test_a_key_far_away(gm, precision):
    """A rare token's key wins over hundreds of others, at the start of the sequence and at tile borders, in prompts and
    in decoding."""
    config = syn.tufirax_config(48, 40, [attention(2, 1, 24, 0.6, 25.0, 4, 100.0)] * 2)
    bits, weights = seeking_weights(gm, config, 6)
    plan = gm.Model.described(config, bits, 420, 8, precision)
    askers = np.array([150, 299, 419])
    for place in (0, 1, 31, 32, 63, 64, 127, 128):
        tokens = tokens_for(config, 420, place) % 38
        tokens[place], tokens[askers] = 38, 39
        want, limits = plain(config, weights, tokens, precision)
        other = tokens.copy()
        other[place] = 5
        assert (row_errors(o.Reference(config, weights).extend(other), want)[askers] > 5 * limits[askers]).all()
        plan.reset()
        assert within(plan.extend(tokens, range(420)), want, limits), place
        plan.reset()
        plan.extend(tokens[:400])
        got = [plan.extend(tokens[t:t + 1], [0])[0] for t in range(400, 420)]
        assert within(np.stack(got), want[400:], limits[400:]), place


@pytest.mark.parametrize("precision", PRECISIONS)
def test_keys_inside_a_portion(gm, precision):
    """The key lies among the portion's own rows or right before them: every distance over the border between what is
    cached and what the pass brings."""
    config = syn.tufirax_config(48, 40, [attention(2, 1, 24, 0.6, 25.0, 4, 100.0)])
    bits, weights = seeking_weights(gm, config, 7)
    plan = gm.Model.described(config, bits, 128, 8, precision)
    for place, asker in ((60, 61), (61, 66), (63, 64), (64, 65), (66, 69), (71, 71 + 9), (40, 66)):
        tokens = tokens_for(config, 90, place) % 38
        tokens[place], tokens[asker] = 38, 39
        want, limits = plain(config, weights, tokens, precision)
        other = tokens.copy()
        other[place] = 5
        assert row_errors(o.Reference(config, weights).extend(other), want)[asker] > 5 * limits[asker]
        for cuts in ((64, 8, 18), (61, 2, 1, 8, 18), (62, 28), (30, 30, 5, 5, 5, 15)):
            plan.reset()
            at, rows = 0, []
            for size in cuts:
                rows.append(plan.extend(tokens[at:at + size], range(size)))
                at += size
            assert within(np.concatenate(rows), want, limits), (place, asker, cuts)


@pytest.mark.parametrize("precision", PRECISIONS)
def test_a_state_that_hardly_decays(gm, precision):
    """A token's trace in a slow head's state shows hundreds of tokens later, whichever way the prompt is cut."""
    config = syn.tufirax_config(32, 40, [state_space(2, 8, 12, 1, 4, 2)])
    bits, _ = weights_for(gm, config, 9)
    bits["l0.mix.A_log"], bits["l0.mix.dt_bias"] = gm.bf16_bits(np.array([-9.0, -7.0])), gm.bf16_bits(np.array([-1.0, 0.5]))
    weights = {k: gm.bf16_values(v) for k, v in bits.items()}
    tokens = tokens_for(config, 700, 4) % 38
    tokens[3] = 39
    want, limits = plain(config, weights, tokens, precision)
    other = tokens.copy()
    other[3] = 5
    assert row_errors(o.Reference(config, weights).extend(other)[600:], want[600:]).max() > 1e-3
    plan = gm.Model.described(config, bits, 700, 8, precision)
    assert within(plan.extend(tokens, range(700)), want, limits)
    plan.reset()
    plan.extend(tokens[:2])
    plan.extend(tokens[2:650])
    got = [plan.extend(tokens[t:t + 1], [0])[0] for t in range(650, 700)]
    assert within(np.stack(got), want[650:], limits[650:])


# ------------------------------------------------------------------------------------------- batches

@pytest.mark.parametrize("name", ["shared in turn", "states and feed-forwards"])
@pytest.mark.parametrize("precision", PRECISIONS)
def test_streams_equal_conversations_alone(gm, name, precision):
    """Unequal conversations decoded together, in groups smaller than their number; a slot given back and used again."""
    config, bits, weights = make(gm, name)
    plan = gm.Model.described(config, bits, 160, 4, precision)
    own = tokens_for(config, 30, 50)
    plan.extend(own)                            # the plan's own conversation goes on behind the streams'
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
    streams.release(5)
    for count in (2, 21):                       # nothing of the slot's last conversation shows in the next one
        short = tokens_for(config, count, 77)
        again = streams.extend(5, short, range(count))
        assert within(again, *plain(config, weights, short, precision))
        if count == 2:
            streams.release(5)
    assert [streams.position(s) for s in range(6)] == [p.size + 12 for p in prompts[:5]] + [21]
    streams.decode(feeds[0])
    want, limits = plain(config, weights, np.concatenate([prompts[2], feeds[:, 2], feeds[0, 2:3]]), precision)
    assert within(streams.logits(2)[None], want[-1:], limits[-1:])
    # portions of one stream between the others' steps, decoding on behind them
    extra = tokens_for(config, 11, 78)
    streams.extend(5, extra[:5])
    got = np.concatenate([streams.extend(5, extra[5:7], [0, 1]), streams.extend(5, extra[7:], [0, 3])])
    want, limits = plain(config, weights, np.concatenate([short, feeds[0, 5:6], extra]), precision)
    assert within(got, want[[27, 28, 29, 32]], limits[[27, 28, 29, 32]])
    assert plan.position == 30
    tail = tokens_for(config, 9, 51)
    want, limits = plain(config, weights, np.concatenate([own, tail]), precision)
    assert within(plan.extend(tail, range(9)), want[30:], limits[30:])


@pytest.mark.parametrize("name", ["heads of their own", "shared in turn"])
def test_greedy_generation(gm, name):
    """The generation engine, the batch, the engine with a drafter, and the plain implementation choose the same tokens.
    The drafter is the model with one layer weakened, so that some of its drafts are rejected and its state goes back."""
    from guffin_b200 import engine as ge
    config, bits, weights = make(gm, name, 11)
    plan = gm.Model.described(config, bits, 256, 4, "float32")
    prompts = [tokens_for(config, n, n) for n in (40, 3, 90)]
    wanted = [greedy_reference(o.Reference, config, weights, p, 48) for p in prompts]
    assert all(margin > 1e-3 for _, margin in wanted) and len(set(wanted[0][0])) > 5
    options = ge.sampler_options(0.0)
    engine = ge.H1(plan, None, ge.H1Options(options, 0, 0, 0.0, 0, 0))
    for prompt, (want, _) in zip(prompts, wanted):
        engine.prefill(prompt)
        assert engine.generate(48).tolist() == want
    batch = ge.Batch(plan, prompts, options)
    assert batch.generate(48).tolist() == [want for want, _ in wanted]
    weaker = {k: (gm.bf16_bits(gm.bf16_values(v) * 0.8) if k == "l1.norm1" else v) for k, v in bits.items()}
    for horizon in (1, 3):
        draft = gm.Model.described(config, weaker, 256, 4, "float32")
        speculative = ge.H1(plan, draft, ge.H1Options(options, 1, 0, 0.0, 0, 0, horizon))
        for prompt, (want, _) in zip(prompts, wanted):
            speculative.prefill(prompt)
            assert speculative.generate(48).tolist() == want, horizon
        stats = speculative.stats()
        assert stats.cycles > 0 and stats.accepted_tokens > 0


def test_seeded_sampling_in_a_batch(gm):
    """A stream's sampled tokens are those of the same conversation generated alone with the same seed."""
    from guffin_b200 import engine as ge
    config, bits, _ = make(gm, "shared in turn")
    plan = gm.Model.described(config, bits, 128, 4, "float32")
    prompts = [tokens_for(config, n, n) for n in (11, 40)]
    options = [ge.sampler_options(0.9, 20, seed=s, repetition_penalty=1.1) for s in (1, 2)]
    rows = ge.Batch(plan, prompts, options).generate(24)
    for prompt, option, row in zip(prompts, options, rows):
        engine = ge.H1(plan, None, ge.H1Options(option, 0, 0, 0.0, 0, 0))
        engine.prefill(prompt)
        assert engine.generate(24).tolist() == row.tolist()


def test_readback_and_binding_errors(gm):
    config, bits, _ = make(gm, "shared in turn")
    plan = gm.Model.described(config, bits, 64, 2)
    plan.extend([1, 2, 3])
    rows = np.zeros(4096, np.float32)
    with pytest.raises(Exception, match="recurrent"):
        gm.check(plan.L.gf_model_read_kv(plan.handle, 0, 0, 1, rows.ctypes.data, rows.ctypes.data))
    with pytest.raises(Exception, match="not a recurrent layer"):
        gm.check(plan.L.gf_model_read_state(plan.handle, 1, rows.ctypes.data))
    with pytest.raises(Exception, match="has no tensor 'l2.norm1'"):                # a layer that uses another one's
        gm.Model.described(config, dict(bits, **{"l2.norm1": bits["l0.norm1"]}), 64, 2)
    with pytest.raises(Exception, match="'l0.mix.conv' is not bound"):
        gm.Model.described(config, {k: v for k, v in bits.items() if k != "l0.mix.conv"}, 64, 2)
    with pytest.raises(Exception, match="should have shape"):
        gm.Model.described(config, dict(bits, **{"l0.mix.conv": bits["l0.mix.conv"][:, :2]}), 64, 2)


# ------------------------------------------------------------------------------------------- folders and programs

@pytest.mark.parametrize("precision", PRECISIONS)
def test_trace_replay(gm, tmp_path, precision):
    config, bits, weights = make(gm, "shared in turn")
    write_folder(tmp_path, config, bits)
    requests = {"a": tokens_for(config, 90, 1), "b": tokens_for(config, 33, 2), "c": tokens_for(config, 5, 3)}
    steps, expected, at = [], [], dict.fromkeys(requests, 0)
    for name, size, want in (("a", 50, [0, 49]), ("a", 2, []), ("b", 33, [32, 4]), ("a", 37, [1]), ("a", 1, [0]), ("c", 5, [0, 4])):
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
    config, bits, weights = make(gm, "shared in turn", 11)
    write_folder(tmp_path, config, bits)
    prompt = tokens_for(config, 40, 40)
    want, _ = greedy_reference(o.Reference, config, weights, prompt, 10)
    text = ",".join(str(t) for t in prompt)
    run = lambda *args: subprocess.run([sys.executable, "-m", "guffin_b200", *args], cwd=ROOT, capture_output=True, text=True, timeout=300)
    one = run("generate", "--model", str(tmp_path), "--tokens", text, "--max-tokens", "10", "--dtype", "float32")
    assert one.returncode == 0 and one.stdout.split() == [str(t) for t in want], one.stderr
    two = run("generate", "--model", str(tmp_path), "--tokens", text, "--tokens", "1 2 3", "--max-tokens", "10", "--dtype", "float32")
    assert two.stdout.splitlines()[0].split() == [str(t) for t in want], two.stderr
    info = run("info", str(tmp_path))
    assert info.returncode == 0 and "mamba2" in info.stdout and "tensors of layer 1" in info.stdout
    assert "Tufirax" in run("models").stdout.split()
