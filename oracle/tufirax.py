"""A plain, slow implementation of the Tufirax decoder in NumPy, one function per mechanism.

Test infrastructure only: it shares no code with the product and computes everything in the precision of the
arrays it is given (float64 by default).  `weights` maps tensor names to arrays; linear weights are [out, in].
"""
from __future__ import annotations

import numpy as np


def exact(x):
    return x


def bf16(x):
    """Rounded to bfloat16 (nearest even), in the precision it came in."""
    bits = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((bits + 0x7fff + ((bits >> 16) & 1)) & np.uint32(0xffff0000)).view(np.float32).astype(np.asarray(x).dtype)


def rms_norm(x, gain, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def rms_norm_in_parts(x, gain, parts, eps):
    """Every one of `parts` equal parts of the last axis by its own root mean square."""
    split = x.reshape(*x.shape[:-1], parts, x.shape[-1] // parts)
    return rms_norm(split, 1.0, eps).reshape(x.shape) * gain


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


# ---- attention

def rotate_halves(x, positions, base, dims):
    """x [T, heads, dim]: dimension i of the first `dims` turns together with dimension i + dims / 2."""
    half = dims // 2
    angle = np.asarray(positions, np.float64)[:, None] * np.float64(base) ** (-2.0 * np.arange(half) / max(dims, 1))
    c, s = np.cos(angle)[:, None, :].astype(x.dtype), np.sin(angle)[:, None, :].astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def soft_cap(scores, cap):
    return cap * np.tanh(scores / cap)


def softmax_with_sink(scores, sink):
    """scores [..., keys]; the sink takes part in the denominator only."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def grouped_attention(q, k, v, first, scale, cap, sink):
    """q [T, heads, dim] at positions first.., k and v [S, kv heads, dim] from position 0 on; [T, heads, dim]."""
    T, heads, _ = q.shape
    S, groups = k.shape[:2]
    seen = np.arange(S)[None, :] <= first + np.arange(T)[:, None]
    out = np.empty((T, heads, v.shape[2]), q.dtype)
    for h in range(heads):
        g = h // (heads // groups)
        scores = np.where(seen, soft_cap((q[:, h] @ k[:, g].T) * scale, cap), -np.inf)
        out[:, h] = softmax_with_sink(scores, sink[h]) @ v[:, g]
    return out


# ---- state space

def causal_convolution(x, before, taps, bias):
    """x [T, channels] behind the rows `before` [taps - 1, channels]; the last tap is the current row's."""
    rows = np.concatenate([before, x])
    count = taps.shape[1]
    return sum(rows[j:j + len(x)] * taps[:, j] for j in range(count)) + bias


def state_space_step(state, x, b, c, dt, a_log, skip):
    """state [heads, N, vdim], x [heads, vdim], b and c [heads, N], dt [heads]: (next state, output [heads, vdim])."""
    decay = np.exp(-np.exp(a_log) * dt)
    state = decay[:, None, None] * state + (dt[:, None] * b)[:, :, None] * x[:, None, :]
    return state, np.einsum("hnv,hn->hv", state, c) + skip[:, None] * x


def gated_feed_forward(x, gate, up, down, cast=exact):
    return cast(gelu_tanh(x @ gate.T) * (x @ up.T)) @ down.T


class Reference:
    """A whole model fed in portions; keeps every key, value and state.  `cast` is applied to what enters a matrix
    product or the key/value cache: with bf16 it shows what rounding alone does."""

    def __init__(self, config, weights, dtype=np.float64, cast=exact):
        self.config, self.cast, self.dtype = config, cast, dtype
        self.w = {k: np.asarray(v, dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.position = 0
        self.residuals = []
        self.keys, self.values, self.states, self.inputs = {}, {}, {}, {}

    def owner(self, i):
        """The layer whose tensors layer i uses."""
        while "weights_of" in self.config["layers"][i]:
            i = self.config["layers"][i]["weights_of"]
        return i

    def attention(self, i, x):
        m, w, eps, cast, p = self.config["layers"][i]["mixer"], self.w, self.config["norm"]["eps"], self.cast, f"l{self.owner(i)}.mix"
        T, heads, groups, dim = len(x), m["heads"], m["kv_heads"], m["dim"]
        raw = x @ w[p + ".k"].T
        places = self.position + np.arange(T)
        q = rms_norm(x @ w[p + ".q"].T, w[p + ".q.norm"], eps).reshape(T, heads, dim)
        k = rms_norm(raw, w[p + ".k.norm"], eps).reshape(T, groups, dim)
        q, k = (cast(rotate_halves(a, places, m["rot"]["base"], m["rot"]["dims"])) for a in (q, k))
        v = cast(raw).reshape(T, groups, dim)
        if i in self.keys:
            k, v = np.concatenate([self.keys[i], k]), np.concatenate([self.values[i], v])
        self.keys[i], self.values[i] = k, v
        y = grouped_attention(q, k, v, self.position, m["scale"], m["softcap"], w[p + ".sink"])
        y = y * sigmoid(x @ w[p + ".g"].T)[:, :, None]
        return cast(y.reshape(T, heads * dim)) @ w[p + ".o"].T

    def mamba2(self, i, x):
        m, w, eps, cast, p = self.config["layers"][i]["mixer"], self.w, self.config["norm"]["eps"], self.cast, f"l{self.owner(i)}.mix"
        T, heads, vdim, N, G, taps = len(x), m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
        inner = heads * vdim
        z, xbc, dt = np.split(x @ w[p + ".in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
        before = self.inputs.get(i, np.zeros((taps - 1, xbc.shape[1]), self.dtype))
        self.inputs[i] = np.concatenate([before, xbc])[T:]
        xs, b, c = np.split(silu(causal_convolution(xbc, before, w[p + ".conv"], w[p + ".conv.b"])), [inner, inner + G * N], axis=1)
        dt = softplus(dt + w[p + ".dt_bias"])
        state = self.states.get(i, np.zeros((heads, N, vdim), self.dtype))
        group = np.arange(heads) // (heads // G)
        y = np.empty((T, inner), self.dtype)
        for t in range(T):
            state, out = state_space_step(state, xs[t].reshape(heads, vdim), b[t].reshape(G, N)[group], c[t].reshape(G, N)[group], dt[t],
                                          w[p + ".A_log"], w[p + ".D"])
            y[t] = out.reshape(inner)
        self.states[i] = state
        return cast(rms_norm_in_parts(y * silu(z), w[p + ".norm"], m["norm_groups"], eps)) @ w[p + ".o"].T

    def extend(self, tokens):
        """Logits of every token of the portion; self.residuals holds the stream behind each layer."""
        c, w, eps, cast = self.config, self.w, self.config["norm"]["eps"], self.cast
        x = w["embed"][np.asarray(tokens)]
        self.residuals = []
        for i, layer in enumerate(c["layers"]):
            p = f"l{self.owner(i)}"
            y = (self.attention if layer["type"] == "attention" else self.mamba2)(i, cast(x))
            x = x + rms_norm(y, w[p + ".norm1"], eps)
            if layer.get("mlp"):
                y = gated_feed_forward(cast(x), w[p + ".mlp.gate"], w[p + ".mlp.up"], w[p + ".mlp.down"], cast)
                x = x + rms_norm(y, w[p + ".norm2"], eps)
            self.residuals.append(x)
        self.position += len(tokens)
        return cast(rms_norm(x, w["final.norm"], eps)) @ w["head"].T
