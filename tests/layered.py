"""What the tests of layered designs share: errors of logits, token sequences, model folders."""
import json
import struct

import numpy as np


def rel_l2(got, want):
    return float(np.linalg.norm(np.asarray(got, np.float64) - want) / max(np.linalg.norm(want), 1e-30))


def row_errors(got, want):
    """Per row: root mean square of the difference over that of the wanted logits, means taken off."""
    d, w = np.asarray(got, np.float64) - want, want - want.mean(1, keepdims=True)
    d -= d.mean(1, keepdims=True)
    return np.sqrt((d * d).mean(1) / (w * w).mean(1))


def limits_of(reference, rounding, config, weights, tokens, precision):
    """The plain implementation's logits and the error a row may have: three times what rounding alone causes there, or
    to the worst rows but a few."""
    want = reference(config, weights).extend(tokens)
    if precision == "float32":
        return want, np.full(len(tokens), 1e-4)
    rounded = row_errors(reference(config, weights, cast=rounding).extend(tokens), want)
    return want, 3.0 * np.maximum(rounded, max(np.quantile(rounded, 0.98), 2e-3))


def within(got, want, limits):
    return bool((row_errors(got, want) <= limits).all())


def tokens_for(config, count, seed=0):
    return np.random.default_rng(seed).integers(0, config["vocab"], count).astype(np.uint32)


def write_folder(path, config, bits):
    header, blob = {"__metadata__": {"format": "pt"}}, b""
    for name, value in bits.items():
        header[name] = dict(dtype="BF16", shape=list(value.shape), data_offsets=[len(blob), len(blob) + value.nbytes])
        blob += value.tobytes()
    text = json.dumps(header).encode()
    (path / "config.json").write_text(json.dumps(config))
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + blob)


def greedy_reference(reference, config, weights, prompt, count):
    """(tokens, smallest margin between the best and the second best logit)."""
    ref, out, margins = reference(config, weights), [], []
    logits = ref.extend(prompt)[-1]
    for _ in range(count):
        out.append(int(np.argmax(logits)))
        top = np.sort(logits)[-2:]
        margins.append(top[1] - top[0])
        logits = ref.extend(out[-1:])[-1]
    return out, min(margins)
