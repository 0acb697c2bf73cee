"""Layered decoders on the host: configuration and tensor reading, family selection, trace replay, the oracle itself."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from tests import layered_models as L

ROOT = Path(__file__).resolve().parent.parent


def small():
    return L.model([L.layer(), L.layer(L.mixer(scaling=L.YARN, vdim=36), ff=None), L.layer(weights_of=0)])


def test_artifact_round_trip(tmp_path):
    from stark_b200 import registry
    from stark_b200.artifact import write_layered
    root = small()
    w = L.weights(root)
    write_layered(tmp_path, root, w)
    opened = registry.open_model(tmp_path)
    assert opened.family == "Guvulorn" and opened.vocab == root["vocab"] and "float32" in opened.dtypes
    assert set(opened.weights) == set(w)
    for k in w:
        assert np.array_equal(opened.weights[k], w[k])
    cfg = opened.cfg
    assert [l["weights_of"] for l in cfg["layers"]] == [None, None, 0]
    assert cfg["layers"][1]["ff"] is None and cfg["layers"][1]["rot"]["scaling"]["original"] == 96
    assert cfg["layers"][0]["rot"]["scaling"] is None and cfg["layers"][1]["vdim"] == 36
    assert opened.prompt_scratch_bytes() > 0


@pytest.mark.parametrize("spoil", ["missing", "extra", "shape", "mixer", "kind", "circle"])
def test_artifact_refusals(tmp_path, spoil):
    from stark_b200 import registry
    from stark_b200.artifact import ArtifactError, write_layered
    root = small()
    w = L.weights(root)
    if spoil == "missing":
        del w["l1.mix.uk"]
    elif spoil == "extra":
        w["l1.norm2"] = w["l1.norm1"]
    elif spoil == "shape":
        w["head"] = w["head"][:, :-1].copy()
    elif spoil == "mixer":
        root["layers"][0]["type"] = "something_else"
    elif spoil == "kind":
        root["layers"][0]["mlp"]["kind"] = "routed"
    else:
        root["layers"][2]["weights_of"] = 2
    write_layered(tmp_path, root, w)
    with pytest.raises(ArtifactError):
        registry.open_model(tmp_path)


def test_unknown_architecture(tmp_path):
    from stark_b200 import registry
    from stark_b200.artifact import ArtifactError
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ArtifactError):
        registry.open_model(tmp_path)


def test_weights_of_chain_resolves():
    from stark_b200.artifact import layered_config
    root = L.model([L.layer(), L.layer(weights_of=0), L.layer(weights_of=1)])
    assert [l["weights_of"] for l in layered_config(root)["layers"]] == [None, 0, 0]


def c_load(path) -> int:
    import ctypes as C
    from stark_b200 import _lib
    opts = _lib.LoadOptions(C.sizeof(_lib.LoadOptions), _lib.ABI_VERSION, 64, 0)
    handle = C.c_void_p()
    raw = str(path).encode()
    status = _lib.load().stark_b200_load(raw, len(raw), C.byref(opts), C.byref(handle))
    if handle.value:
        _lib.load().stark_b200_destroy(C.byref(handle))
    return status


@pytest.mark.parametrize("spoil,status", [("missing", 1), ("extra", 1), ("shape", 1), ("mixer", 5), ("kind", 5), ("circle", 1),
                                          ("size", 1), (None, None)])
def test_library_loader_checks_before_it_touches_a_device(tmp_path, spoil, status):
    from stark_b200.artifact import write_layered
    root = small()
    w = L.weights(root)
    if spoil == "missing":
        del w["l1.mix.uk"]
    elif spoil == "extra":
        w["l1.norm2"] = w["l1.norm1"]
    elif spoil == "shape":
        w["head"] = w["head"][:, :-1].copy()
    elif spoil == "mixer":
        root["layers"][0]["type"] = "something_else"
    elif spoil == "kind":
        root["layers"][0]["mlp"]["kind"] = "routed"
    elif spoil == "circle":
        root["layers"][2]["weights_of"] = 2
    elif spoil == "size":
        root["width"] = 80
    write_layered(tmp_path, root, w)
    assert c_load(tmp_path) == status if status is not None else c_load(tmp_path) in (0, 8)  # 8: no device here


class FakeModel:
    def __init__(self):
        self.calls = []

    def reset(self):
        self.calls.append("reset")

    def prefill_rows(self, tokens, rows):
        self.calls.append((list(tokens), list(rows)))
        return np.array([[r, len(tokens)] for r in rows], np.float32).reshape(-1, 2)


def test_trace_replay_order_and_reset():
    from stark_b200.trace import Replay, TraceError
    m = FakeModel()
    r = Replay(m)
    out = np.frombuffer(r.step({"step": 0, "entries": [{"id": "a", "tokens": [4, 5, 6], "want": [2, 0, 2]}]}), "<f4")
    assert out.reshape(-1, 2)[:, 0].tolist() == [2, 0, 2]          # the order asked for, repeats included
    assert r.step({"step": 1, "entries": [{"id": "a", "tokens": [7], "want": []}], "end": ["a"]}) == b""
    r.step({"step": 2, "entries": [{"id": "b", "tokens": [1], "want": [0]}]})
    assert m.calls == ["reset", ([4, 5, 6], [0, 2]), ([7], []), "reset", "reset", ([1], [0])]
    with pytest.raises(TraceError):
        r.step({"step": 3, "entries": [{"id": "c", "tokens": [1], "want": []}]})


def test_trace_run_help():
    out = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--help"], capture_output=True, text=True)
    assert out.returncode == 0 and "--max-tokens" in out.stdout


def test_layered_part_is_a_library_of_its_own():
    import ctypes
    from stark_b200 import build
    lib = ctypes.CDLL(str(build.build(part="layered")))
    for name in ("stark_b200_layered_create", "stark_b200_prefill_rows", "stark_b200_step", "stark_b200_sample",
                 "stark_b200_generate_greedy"):
        assert hasattr(lib, name)
    assert not hasattr(lib, "stark_b200_model_create")


# ------------------------------------------------------------------------------------------------ the oracle itself

def test_oracle_portions_agree():
    root = small()
    w = L.weights(root)
    ids = L.tokens(root, 40)
    whole = L.oracle(root, w).feed(ids)
    for cut in (1, 2, 7):
        o = L.oracle(root, w)
        got = np.concatenate([o.feed(ids[i:i + cut]) for i in range(0, 40, cut)])
        assert np.abs(got - whole).max() < 1e-9


def test_oracle_absorbed_form():
    """The score and output of the cached form (key and value matrices on the query's and output's side)."""
    from oracle import layered as O
    root = small()
    w = {k: L.from_bf16(v).astype(np.float64) for k, v in L.weights(root).items()}
    m = root["layers"][1]["mixer"]
    h = np.random.default_rng(3).standard_normal((9, root["width"]))
    want, (c, r) = O.latent_attention(m, w, "l1.mix", h, 0, None, 1e-5)
    qn, qr = O.latent_queries(m, w, "l1.mix", h, np.arange(9))
    uk = w["l1.mix.uk"].reshape(m["heads"], m["dim"], -1)
    uv = w["l1.mix.uv"].reshape(m["heads"], m["vdim"], -1)
    s = (np.einsum("ihd,hdr,jr->hij", qn, uk, c) + np.einsum("ihd,jd->hij", qr, r)) * m["scale"]
    s = np.where(np.tril(np.ones((9, 9), bool))[None], s, -np.inf)
    a = np.exp(s - s.max(-1, keepdims=True))
    a /= a.sum(-1, keepdims=True)
    got = np.einsum("hij,jr,her->ihe", a, c, uv).reshape(9, -1) @ w["l1.mix.o"].T
    assert np.abs(got - want).max() < 1e-10


def test_oracle_rotation_is_relative_and_scaled():
    from oracle import layered as O
    rot = {"base": 500.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    x = np.random.default_rng(0).standard_normal((1, 12))
    y = np.random.default_rng(1).standard_normal((1, 12))
    f, factor = O.rotary_frequencies(rot)
    assert factor == pytest.approx(0.1 * np.log(4.0) + 1.0)
    assert np.all(f <= 500.0 ** (-np.arange(0, 8, 2) / 8) + 1e-15) and f[0] == 1.0
    a = (O.rotate(x, [7], rot)[0, :8] * O.rotate(y, [3], rot)[0, :8]).sum()
    b = (O.rotate(x, [104], rot)[0, :8] * O.rotate(y, [100], rot)[0, :8]).sum()
    assert a == pytest.approx(b)
    assert np.array_equal(O.rotate(x, [7], rot)[0, 8:], x[0, 8:])


def test_oracle_bigram_rows():
    from oracle import layered as O
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert O.bigram_rows([4, 5, 4], b) == [10, (12 + 35) % 10, (15 + 28) % 10]


def test_oracle_clamps():
    from oracle import layered as O
    assert O.clamped_gate(np.array(9.0), np.array(-9.0), 1.5) == pytest.approx(1.5 / (1 + np.exp(-1.702 * 1.5)) * (-1.5 + 1))
    assert O.clamped_gate(np.array(-9.0), np.array(9.0), 1.5) == pytest.approx(-9.0 / (1 + np.exp(1.702 * 9.0)) * 2.5)
