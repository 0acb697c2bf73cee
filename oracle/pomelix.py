"""Plain restatement of a Pomelix decoder on the CPU: test infrastructure, never on the product path.

One function per mechanism, every one a direct transcription of its equation in numpy, in the precision of its inputs
(float64 in the tests).  ``config`` is the parsed ``config.json``; ``weights`` maps tensor names to arrays.  Nothing
here is shared with the engine.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    return x / rms(x, eps) * w


def short_convolution(u, w, past):
    """Causal convolution over time per channel: row t is sum_j w[:, j] u[t - taps + 1 + j].  ``past`` holds the
    taps - 1 rows that came before ``u``, zeros where there were none."""
    taps = w.shape[1]
    rows = np.concatenate([past, u])
    out = np.zeros_like(u)
    for t in range(len(u)):
        for j in range(taps):
            out[t] += w[:, j] * rows[t + j]
    return out


def query_temperature(position, coef, every):
    return 1.0 + coef * np.log((int(position) + 1) // int(every) + 1)


def mixed_values(v, first, share):
    return (1.0 - share) * v + share * first


def grouped_attention(q, keys, values, first_pos, scale):
    """q [rows, heads, dim] at positions first_pos.. over keys [n, groups, dim] and values [n, groups, vdim]; heads /
    groups neighbouring query heads share a group.  A row attends to the keys up to and including its own position."""
    per = q.shape[1] // keys.shape[1]
    out = np.zeros((q.shape[0], q.shape[1], values.shape[2]), q.dtype)
    for h in range(q.shape[1]):
        g = h // per
        for i in range(len(q)):
            n = first_pos + i + 1
            s = keys[:n, g] @ q[i, h] * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ values[:n, g]
    return out


def silu(z):
    return z / (1.0 + np.exp(-z))


def feed_forward(weights, p, h):
    return (silu(h @ weights[p + ".gate"].T) * (h @ weights[p + ".up"].T)) @ weights[p + ".down"].T


class Mixer:
    """One layer's attention and its state: past projected rows of the convolutions, normed keys, (mixed) values."""

    def __init__(self, mixer, weights, p, eps, first_mixed):
        self.m, self.w, self.p, self.eps, self.first_mixed = mixer, weights, p, eps, first_mixed
        self.past = {}
        self.keys = self.values = None

    def projected(self, name, h):
        u = h @ self.w[self.p + "." + name].T
        w = self.w[self.p + "." + name + ".conv"]
        past = self.past.get(name, np.zeros((w.shape[1] - 1, u.shape[1]), u.dtype))
        out = short_convolution(u, w, past)
        self.past[name] = np.concatenate([past, u])[len(u):]
        return out

    def __call__(self, h, first_pos, shared):
        m, n = self.m, len(h)
        q = self.projected("q", h).reshape(n, m["heads"], m["dim"])
        k = self.projected("k", h).reshape(n, m["kv_heads"], m["dim"])
        v = self.projected("v", h).reshape(n, m["kv_heads"], m["vdim"])
        q, k = q / rms(q, self.eps), k / rms(k, self.eps)
        for i in range(n):
            q[i] *= query_temperature(first_pos + i, m["q_temp"]["coef"], m["q_temp"]["every"])
        if m["v_mix"]:
            if self.first_mixed:
                shared["v"] = v
            else:
                v = mixed_values(v, shared["v"].reshape(v.shape), self.w[self.p + ".vmix"])
        self.keys = k if self.keys is None else np.concatenate([self.keys, k])
        self.values = v if self.values is None else np.concatenate([self.values, v])
        out = grouped_attention(q, self.keys, self.values, first_pos, m["scale"])
        return out.reshape(n, -1) @ self.w[self.p + ".o"].T


class PomelixOracle:
    """A sequence fed in portions of any size; ``feed`` returns the logits of every row it was given."""

    def __init__(self, config, weights, dtype=np.float64):
        self.config = config
        self.weights = {k: np.asarray(v, dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        eps, seen, self.mixers = self.config["norm"]["eps"], False, []
        for i, layer in enumerate(self.config["layers"]):
            mixes = bool(layer["mixer"]["v_mix"])
            self.mixers.append(Mixer(layer["mixer"], self.weights, "l%d.mix" % i, eps, mixes and not seen))
            seen = seen or mixes
        self.position = 0
        self.streams = []

    def feed(self, tokens):
        cfg, w, eps = self.config, self.weights, self.config["norm"]["eps"]
        x = w["embed"][np.asarray(tokens, np.int64)]
        self.streams, shared = [], {}
        for i, layer in enumerate(cfg["layers"]):
            p = "l%d" % i
            h = norm(x, w[p + ".norm1"], eps)
            y = self.mixers[i](h, self.position, shared) * w[p + ".ls1"]
            if layer["mlp"] is not None:
                y = y + feed_forward(w, p + ".mlp", h) * w[p + ".ls2"]
            x = x + cfg["residual_mult"] * y
            self.streams.append(x)
        self.position += len(tokens)
        return norm(x, w["final.norm"], eps) @ w["embed"].T
