"""Plain restatement of a layered decoder (Guvulorn) on the CPU: test infrastructure, never on the product path.

One function per mechanism, every one a direct transcription of its equation in numpy, in the precision of its inputs
(float64 in the tests).  ``config`` is the parsed ``config.json``; ``weights`` maps tensor names to arrays.  Nothing
here is shared with the engine.
"""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_one(x, w, eps):
    """x / rms(x) * (1 + w)"""
    return x / rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return x / rms(x, eps) * w


def bigram_rows(tokens, bigram):
    """Row of the bigram table per token: a hash of (previous, current); the last row where there is no previous."""
    rows = []
    for i, t in enumerate(tokens):
        if i == 0:
            rows.append(bigram["buckets"])
        else:
            rows.append((int(tokens[i - 1]) * bigram["mul_prev"] + int(t) * bigram["mul_cur"]) % bigram["buckets"])
    return rows


def embedding(config, weights, tokens):
    e = config["embedding"]
    x = weights["embed"][np.asarray(tokens)] * e["scale"]
    x = x + weights["bigram"][np.asarray(bigram_rows(tokens, e["bigram"]))]
    return norm_around_one(x, weights["embed.norm"], config["norm"]["eps"])


def rotary_frequencies(rot):
    """(frequency per pair, factor on cos and sin)"""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(s["fast"])), 0)
    hi = min(math.ceil(dim_of(s["slow"])), dims - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)])
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """Interleaved pairs (2i, 2i + 1) of the first ``dims`` entries of the last axis; x is [rows, ..., width]."""
    f, factor = rotary_frequencies(rot)
    angle = np.asarray(positions, np.float64)[:, None] * f[None, :]
    shape = (angle.shape[0],) + (1,) * (x.ndim - 2) + (angle.shape[1],)
    c, s = (np.cos(angle) * factor).reshape(shape), (np.sin(angle) * factor).reshape(shape)
    out = np.array(x)
    d = rot["dims"]
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    out[..., 0:d:2] = u * c - v * s
    out[..., 1:d:2] = v * c + u * s
    return out


def latent_rows(mixer, weights, p, h, positions, eps):
    """What a layer caches per row: (normed latent, rotated shared key part)."""
    rank = mixer["kv_rank"]
    z = h @ weights[p + ".dkv"].T
    return norm_plain(z[:, :rank], weights[p + ".dkv.norm"], eps), rotate(z[:, rank:], positions, mixer["rot"])


def latent_queries(mixer, weights, p, h, positions):
    dim, rd, heads = mixer["dim"], mixer["rot_dim"], mixer["heads"]
    q = (h @ weights[p + ".q"].T).reshape(len(h), heads, dim + rd)
    return q[..., :dim], rotate(q[..., dim:], positions, mixer["rot"])


def latent_attention(mixer, weights, p, h, first_pos, cache, eps):
    """Rows h at positions first_pos.. over the cached (latent, rotated key) rows plus their own; returns the output
    rows and the grown cache."""
    dim, vdim, heads, rank = mixer["dim"], mixer["vdim"], mixer["heads"], mixer["kv_rank"]
    positions = first_pos + np.arange(len(h))
    qn, qr = latent_queries(mixer, weights, p, h, positions)
    c_new, r_new = latent_rows(mixer, weights, p, h, positions, eps)
    c = c_new if cache is None else np.concatenate([cache[0], c_new])
    r = r_new if cache is None else np.concatenate([cache[1], r_new])
    keys = (c @ weights[p + ".uk"].T).reshape(len(c), heads, dim)
    values = (c @ weights[p + ".uv"].T).reshape(len(c), heads, vdim)
    score = (np.einsum("ihd,jhd->hij", qn, keys) + np.einsum("ihd,jd->hij", qr, r)) * mixer["scale"]
    visible = np.arange(len(c))[None, :] <= positions[:, None]
    score = np.where(visible[None], score, -np.inf)
    e = np.exp(score - score.max(axis=-1, keepdims=True))
    a = e / e.sum(axis=-1, keepdims=True)
    out = np.einsum("hij,jhe->ihe", a, values).reshape(len(h), heads * vdim)
    return out @ weights[p + ".o"].T, (c, r)


def clamped_gate(g, u, limit):
    g = np.minimum(g, limit)
    u = np.clip(u, -limit, limit)
    return g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)


def feed_forward(mlp, weights, p, h):
    g = h @ weights[p + ".gate"].T + weights[p + ".gate.b"]
    u = h @ weights[p + ".up"].T + weights[p + ".up.b"]
    return clamped_gate(g, u, mlp["limit"]) @ weights[p + ".down"].T + weights[p + ".down.b"]


class LayeredOracle:
    """A sequence fed in portions of any size; ``feed`` returns the logits of every row it was given."""

    def __init__(self, config, weights, dtype=np.float64):
        self.config = config
        self.weights = {k: np.asarray(v, dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.tokens = []
        self.caches = [None] * len(self.config["layers"])
        self.streams = []

    def feed(self, tokens):
        cfg, w, eps = self.config, self.weights, self.config["norm"]["eps"]
        first = len(self.tokens)
        self.tokens += [int(t) for t in tokens]
        x = embedding(cfg, w, self.tokens)[first:]     # the first row's previous token is the last one fed before
        self.streams = []
        for i, layer in enumerate(cfg["layers"]):
            p = "l%d" % layer.get("weights_of", i)
            y, self.caches[i] = latent_attention(layer["mixer"], w, p + ".mix", x, first, self.caches[i], eps)
            x = x + norm_around_one(y, w[p + ".norm1"], eps)
            if layer.get("mlp") is not None:
                x = x + norm_around_one(feed_forward(layer["mlp"], w, p + ".mlp", x), w[p + ".norm2"], eps)
            self.streams.append(x)
        return norm_around_one(x, w["final.norm"], eps) @ w["head"].T
