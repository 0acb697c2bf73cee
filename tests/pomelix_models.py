"""Small Pomelix decoders with random weights for the tests: configurations in the form of their config.json, weights as
bf16 bit patterns, the oracle over the same values."""
from __future__ import annotations

import numpy as np

from oracle.pomelix import PomelixOracle
from tests.layered_models import LIMIT, engine, error, from_bf16, to_bf16, tokens  # noqa: F401


def mixer(heads=6, kv_heads=2, dim=20, vdim=28, conv=4, scale=0.4, coef=0.5, every=24, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
            "q_temp": {"coef": coef, "every": every}, "v_mix": v_mix}


def layer(mix=None, ff=40):
    return {"type": "attention", "mixer": mix or mixer(), "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(layers, vocab=75, width=72, residual_mult=0.7, eps=3e-5):
    return {"architecture": "Pomelix", "vocab": vocab, "width": width, "residual_mult": residual_mult, "norm": {"eps": eps},
            "layers": layers}


def shapes(root):
    V, D = root["vocab"], root["width"]
    out = {"embed": (V, D), "final.norm": (D,)}
    for i, l in enumerate(root["layers"]):
        m, p = l["mixer"], f"l{i}"
        H, G, dim, vd, taps = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        out.update({p + ".norm1": (D,), p + ".ls1": (D,), p + ".mix.q": (H * dim, D), p + ".mix.k": (G * dim, D),
                    p + ".mix.v": (G * vd, D), p + ".mix.o": (D, H * vd), p + ".mix.q.conv": (H * dim, taps),
                    p + ".mix.k.conv": (G * dim, taps), p + ".mix.v.conv": (G * vd, taps)})
        if m["v_mix"]:
            out[p + ".mix.vmix"] = ()
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            out.update({p + ".ls2": (D,), p + ".mlp.gate": (F, D), p + ".mlp.up": (F, D), p + ".mlp.down": (D, F)})
    return out


def weights(root, seed=0, **override):
    """bf16 bit patterns by name.  ``override``: tensor-name suffix (dots as underscores) -> constant or array."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(root).items():
        if name.endswith(("norm", "norm1", "ls1", "ls2")):
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif name.endswith("vmix"):
            a = rng.uniform(0.2, 0.7)
        elif name.endswith(".conv"):
            a = rng.standard_normal(shape) * 0.4
            a[:, -1] += 0.7
        elif name == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
        for key, value in override.items():
            if name.replace(".", "_").endswith(key):
                a = np.broadcast_to(np.asarray(value, np.float64), shape)
        out[name] = to_bf16(np.asarray(a)).reshape(shape)
    return out


def oracle(root, w):
    return PomelixOracle(root, {k: from_bf16(v).reshape(v.shape) for k, v in w.items()})
