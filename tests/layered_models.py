"""Small layered decoders with random weights for the tests: configurations in the form of their config.json, weights as
bf16 bit patterns, the oracle over the same values."""
from __future__ import annotations

import numpy as np

from oracle.layered import LayeredOracle


def to_bf16(a) -> np.ndarray:
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(b) -> np.ndarray:
    return (np.asarray(b, np.uint16).astype(np.uint32) << 16).view(np.float32)


def mixer(heads=2, dim=24, rot_dim=12, vdim=20, kv_rank=28, scale=0.05, base=10000.0, dims=None, scaling=None):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling:
        rot["scaling"] = scaling
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": rot}


def layer(mix=None, ff=40, limit=2.0, weights_of=None):
    m = mix or mixer()
    e = {"type": "latent_attention" if "scaling" in m["rot"] else "latent_attention_2", "mixer": m,
         "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


YARN = {"factor": 5.0, "original": 96, "fast": 16.0, "slow": 1.5}


def model(layers, vocab=75, width=72, buckets=53, mul_prev=19, mul_cur=5, scale=3.5, eps=3e-5):
    return {"architecture": "Guvulorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": layers}


def shapes(root):
    V, D, B = root["vocab"], root["width"], root["embedding"]["bigram"]["buckets"]
    out = {"embed": (V, D), "bigram": (B + 1, D), "embed.norm": (D,), "final.norm": (D,), "head": (V, D)}
    for i, l in enumerate(root["layers"]):
        if "weights_of" in l:
            continue
        m, p = l["mixer"], f"l{i}"
        H, dim, rd, vd, r = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        out.update({p + ".norm1": (D,), p + ".mix.q": (H * (dim + rd), D), p + ".mix.dkv": (r + rd, D),
                    p + ".mix.dkv.norm": (r,), p + ".mix.uk": (H * dim, r), p + ".mix.uv": (H * vd, r),
                    p + ".mix.o": (D, H * vd)})
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            out.update({p + ".norm2": (D,), p + ".mlp.gate": (F, D), p + ".mlp.gate.b": (F,), p + ".mlp.up": (F, D),
                        p + ".mlp.up.b": (F,), p + ".mlp.down": (D, F), p + ".mlp.down.b": (D,)})
    return out


def weights(root, seed=0, **override):
    """bf16 bit patterns by name.  ``override``: tensor-name suffix (dots as underscores) -> constant or array."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(root).items():
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            a = 0.3 * rng.standard_normal(shape) + (1.0 if name.endswith("dkv.norm") else 0.0)
        elif len(shape) == 1:
            a = 0.4 * rng.standard_normal(shape)
        elif name in ("embed", "bigram"):
            a = rng.standard_normal(shape) * (0.5 if name == "embed" else 1.5)
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
        for key, value in override.items():
            if name.replace(".", "_").endswith(key):
                a = np.broadcast_to(np.asarray(value, np.float64), shape)
        out[name] = to_bf16(a)
    return out


def oracle(root, w):
    return LayeredOracle(root, {k: from_bf16(v) for k, v in w.items()})


def engine(root, w, context, dtype):
    from stark_b200.artifact import layered_config
    from stark_b200.engine import LayeredModel
    return LayeredModel.load(layered_config(root), w, context, dtype)


def tokens(root, n, seed=1):
    return np.random.default_rng(seed).integers(0, root["vocab"], n).astype(np.uint32)


def error(got, want):
    """Per row: root mean square of the centred difference over the spread of the wanted logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


LIMIT = {"float32": 3e-5, "bfloat16": 0.05}
