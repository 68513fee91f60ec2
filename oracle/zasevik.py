"""A plain, slow implementation of the Zasevik decoder in NumPy, one function per mechanism.

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


def centred_rms_norm(x, weight, eps):
    """The gain is one plus the stored weight."""
    return rms_norm(x, 1.0 + weight, eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def clamped_gate(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def softmax_with_sink(scores, sink):
    """scores [..., keys]; the sink takes part in the denominator only."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def latent(h, down, gain, eps):
    return rms_norm(h @ down.T, gain, eps)


def latent_attention(q, c, first, heads, up_k, up_v, sink, scale, cast=exact):
    """q [T, heads * dim] at positions first.., c [S, rank] every latent from position 0 on; returns [T, heads * vdim]."""
    T, S = q.shape[0], c.shape[0]
    dim, vdim = q.shape[1] // heads, up_v.shape[0] // heads
    k = cast(c @ up_k.T).reshape(S, heads, dim)
    v = cast(c @ up_v.T).reshape(S, heads, vdim)
    q = cast(q).reshape(T, heads, dim)
    seen = np.arange(S)[None, :] <= first + np.arange(T)[:, None]
    out = np.empty((T, heads, vdim), q.dtype)
    for n in range(heads):
        scores = np.where(seen, (q[:, n] @ k[:, n].T) * scale, -np.inf)
        out[:, n] = cast(softmax_with_sink(scores, sink[n])) @ v[:, n]
    return out.reshape(T, heads * vdim)


def dense_feed_forward(h, up, down, cast=exact):
    return cast(squared_relu(h @ up.T)) @ down.T


def expert(h, gate, up, down, limit, cast=exact):
    return cast(clamped_gate(h @ gate.T, h @ up.T, limit)) @ down.T


def route(h, router, top):
    """(chosen experts, their scores) per token: the largest sigmoid scores, the lower index first among equals."""
    scores = sigmoid(h @ router.T)
    chosen = np.argsort(-scores, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(scores, chosen, axis=-1)


def mixture(h, weights, prefix, spec, cast=exact):
    chosen, scores = route(h, weights[prefix + ".router"], spec["router"]["top"])
    limit = spec["expert"]["limit"]
    out = np.zeros((h.shape[0], h.shape[1]), h.dtype)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], scores[t]):
            p = f"{prefix}.e{e}"
            out[t] += expert(s * h[t:t + 1], weights[p + ".gate"], weights[p + ".up"], weights[p + ".down"], limit, cast)[0]
    if spec.get("shared"):
        p = prefix + ".shared"
        y = expert(h, weights[p + ".gate"], weights[p + ".up"], weights[p + ".down"], spec["shared"]["limit"], cast)
        out += sigmoid(h @ weights[p + ".sg"].T) * y
    return out


class Reference:
    """A whole model fed in portions; keeps every latent it has seen.  `cast` is applied to what enters a matrix product
    or the cache: with bf16 it shows what rounding alone does."""

    def __init__(self, config, weights, dtype=np.float64, cast=exact):
        self.config, self.cast = config, cast
        self.w = {k: np.asarray(v, dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.latents = [None] * len(self.config["layers"])
        self.position = 0
        self.residuals = []

    def extend(self, tokens):
        """Logits of every token of the portion; self.residuals holds the stream behind each layer."""
        c, w, eps, cast = self.config, self.w, self.config["norm"]["eps"], self.cast
        x = w["embed"][np.asarray(tokens)] * c["embedding"]["scale"]
        self.residuals = []
        for i, layer in enumerate(c["layers"]):
            p, m = f"l{i}", layer["mixer"]
            h = cast(centred_rms_norm(x, w[p + ".norm1"], eps))
            new = cast(latent(h, w[p + ".mix.dkv"], w[p + ".mix.dkv.norm"], eps))
            self.latents[i] = new if self.latents[i] is None else np.concatenate([self.latents[i], new])
            y = cast(latent_attention(h @ w[p + ".mix.q"].T, self.latents[i], self.position, m["heads"], w[p + ".mix.uk"],
                                      w[p + ".mix.uv"], w[p + ".mix.sink"], m["scale"], cast)) @ w[p + ".mix.o"].T
            x = x + centred_rms_norm(y, w[p + ".norm1b"], eps) * w[p + ".ls1"]
            if layer.get("mlp"):
                h = cast(centred_rms_norm(x, w[p + ".norm2"], eps))
                if layer["mlp"]["kind"] == "dense":
                    y = dense_feed_forward(h, w[p + ".mlp.up"], w[p + ".mlp.down"], cast)
                else:
                    y = mixture(h, w, p + ".mlp", layer["mlp"], cast)
                x = x + centred_rms_norm(y, w[p + ".norm2b"], eps) * w[p + ".ls2"]
            self.residuals.append(x)
        self.position += len(tokens)
        return cast(centred_rms_norm(x, w["final.norm"], eps)) @ w["embed"].T
