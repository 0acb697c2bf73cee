"""Which model family serves a model directory: ``config.json`` decides, as it does in the C loader (``load.cu``).

``open_model(path)`` reads the directory and returns an ``OpenedModel`` -- the configuration, the weights, and how to put
them on the device -- without touching a GPU.  A new family is one entry of ``FAMILIES``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Callable

from .artifact import LAYERED_ARCHITECTURES, ArtifactError, read_artifact, read_layered


@dataclass
class OpenedModel:
    family: str
    cfg: dict
    weights: dict
    vocab: int
    max_context: int            # positions the model's own configuration allows
    root: dict                  # config.json
    dtypes: tuple               # precisions the family serves
    _load: Callable = field(repr=False)
    _scratch: Callable = field(repr=False)

    def load(self, context_tokens: int, dtype: str | None = None):
        """The model on the device, ready for ``prefill``."""
        dtype = dtype or self.dtypes[0]
        if dtype not in self.dtypes:
            raise ArtifactError(f"the {self.family} family does not serve {dtype}")
        return self._load(self.cfg, self.weights, context_tokens, dtype)

    def prompt_scratch_bytes(self, drafts: int = 0) -> int:
        """Device memory a prompt pass may still allocate beyond the cache: its rows of every intermediate."""
        return self._scratch(self.cfg, drafts)


PASS_ROWS = 4096


def _dense_load(cfg, weights, context_tokens, dtype):
    from .engine import DenseModel
    return DenseModel.load(cfg, weights, context_tokens=context_tokens)


def _dense_scratch(c: dict, drafts: int) -> int:
    qkv = (c["q_heads"] + 2 * c["kv_heads"]) * c["head_dim"]
    scratch = PASS_ROWS * 2 * (2 * c["hidden"] + qkv + c["q_heads"] * c["head_dim"] + c["inter"])
    if drafts:
        scratch += 16 * 2 * (c["vocab"] + 4 * c["hidden"])
    return scratch


def _open_dense(path: Path, root: dict) -> OpenedModel:
    cfg, weights = read_artifact(path)
    try:
        layer0 = root["decoder_config"]["transformer_config"]["layer_configs"][0]
        limit = int(layer0["rope_config"].get("max_sequence_length") or 32768)
    except (KeyError, IndexError, TypeError, ValueError):
        limit = 32768
    return OpenedModel("dense", cfg, weights, cfg["vocab"], limit, root, ("bfloat16",), _dense_load, _dense_scratch)


def _layered_load(cfg, weights, context_tokens, dtype):
    from .engine import LayeredModel
    return LayeredModel.load(cfg, weights, context_tokens, dtype)


def _layered_scratch(c: dict, drafts: int) -> int:
    pad = lambda n: -(-n // 64) * 64
    widest = lambda f: max(f(l) for l in c["layers"])

    def projected(l):
        if l["mixer"] == "latent":
            return l["heads"] * (pad(l["dim"]) + pad(l["rot_dim"])) + pad(l["kv_rank"]) + pad(l["rot_dim"])
        return 2 * l["heads"] * pad(l["dim"]) + l["kv_heads"] * (pad(l["dim"]) + 3 * pad(l["vdim"]))

    row = 2 * (pad(c["width"]) * 5 + widest(projected)
               + widest(lambda l: l["heads"] * pad(l["vdim"])) + widest(lambda l: pad(l["ff"]["width"]) if l["ff"] else 64)
               + widest(lambda l: l["heads"] * (pad(l["dim"]) + pad(l["vdim"])) if l["mixer"] == "latent" else 0) * 3 // 2)
    return PASS_ROWS * row + 128 * 4 * c["vocab"]


def _open_layered(path: Path, root: dict) -> OpenedModel:
    cfg, weights = read_layered(path)
    # the configuration sets no limit on positions; the angles stay exact in f32 far beyond this
    return OpenedModel(cfg["architecture"], cfg, weights, cfg["vocab"], 1 << 20, root, ("bfloat16", "float32"), _layered_load,
                       _layered_scratch)


# (does this family's config.json look like that, how to open it)
FAMILIES: list[tuple[Callable[[dict], bool], Callable[[Path, dict], OpenedModel]]] = [
    (lambda root: root.get("type") == "LanguageModelConfig", _open_dense),
    (lambda root: root.get("architecture") in LAYERED_ARCHITECTURES, _open_layered),
]


def open_model(path) -> OpenedModel:
    path = Path(path)
    root = json.loads((path / "config.json").read_text())
    if not isinstance(root, dict):
        raise ArtifactError("config.json is not an object")
    for matches, opener in FAMILIES:
        if matches(root):
            return opener(path, root)
    raise ArtifactError(f"no model family serves type {root.get('type')!r}, architecture {root.get('architecture')!r}")
