"""Pomelix on the host: configuration and tensor reading, refusals by both readers, the oracle against itself."""
import numpy as np
import pytest

from tests import pomelix_models as P
from tests.test_layered_host import c_load


def small():
    return P.model([P.layer(), P.layer(P.mixer(heads=4, kv_heads=4, conv=2, v_mix=False), ff=None), P.layer(ff=33)])


def test_artifact_round_trip(tmp_path):
    from stark_b200 import registry
    from stark_b200.artifact import write_layered
    root = small()
    w = P.weights(root)
    write_layered(tmp_path, root, w)
    opened = registry.open_model(tmp_path)
    assert opened.family == "Pomelix" and opened.vocab == root["vocab"] and "float32" in opened.dtypes
    assert set(opened.weights) == set(w)
    for k in w:
        assert np.array_equal(opened.weights[k], w[k])
    cfg = opened.cfg
    assert cfg["arrangement"] == "parallel" and cfg["tied"] and not cfg["embed_norm"] and cfg["residual_mult"] == 0.7
    assert [l["v_mix"] for l in cfg["layers"]] == [True, False, True] and cfg["layers"][1]["ff"] is None
    assert cfg["layers"][0]["q_temp"] == dict(coef=0.5, every=24) and cfg["layers"][1]["conv"] == 2
    assert opened.prompt_scratch_bytes() > 0


def test_optional_parts(tmp_path):
    from stark_b200 import registry
    from stark_b200.artifact import write_layered
    root = small()
    w = P.weights(root)
    m = root["layers"][1]["mixer"]
    del m["v_mix"]
    m["q_temp"] = m["conv"] = None
    for name in list(w):
        if name.startswith("l1.mix") and name.endswith("conv"):
            del w[name]
    w["l1.mix.vmix"] = w["l0.mix.vmix"]          # a share nobody uses
    write_layered(tmp_path, root, w)
    layer = registry.open_model(tmp_path).cfg["layers"][1]
    assert layer["conv"] == 0 and layer["q_temp"] is None and layer["v_mix"] is False
    assert c_load(tmp_path) in (0, 8)            # 8: no device here


SPOILS = {"missing": 1, "extra": 1, "shape": 1, "taps": 1, "head": 1, "mixer": 5, "kind": 5, "groups": 1, "every": 1, "scalar": 1}


@pytest.mark.parametrize("spoil", SPOILS)
def test_refusals(tmp_path, spoil):
    from stark_b200 import registry
    from stark_b200.artifact import ArtifactError, write_layered
    root = small()
    w = P.weights(root)
    if spoil == "missing":
        del w["l2.ls2"]
    elif spoil == "extra":
        w["l1.ls2"] = w["l0.ls2"]                # a layer without a feed-forward
    elif spoil == "shape":
        w["l0.mix.v"] = w["l0.mix.v"][:-1].copy()
    elif spoil == "taps":
        root["layers"][0]["mixer"]["conv"] = 3
    elif spoil == "head":
        w["head"] = w["embed"]                   # the read-out is the embedding
    elif spoil == "mixer":
        root["layers"][0]["type"] = "attention_2"
    elif spoil == "kind":
        root["layers"][0]["mlp"]["kind"] = "routed"
    elif spoil == "groups":
        root["layers"][0]["mixer"]["kv_heads"] = 4
    elif spoil == "every":
        root["layers"][0]["mixer"]["q_temp"]["every"] = 0
    else:
        w["l0.mix.vmix"] = w["l0.mix.vmix"].reshape(1)
    write_layered(tmp_path, root, w)
    with pytest.raises(ArtifactError):
        registry.open_model(tmp_path)
    assert c_load(tmp_path) == SPOILS[spoil]


# ------------------------------------------------------------------------------------------------ the oracle itself

def test_oracle_portions_agree():
    root = small()
    w = P.weights(root)
    ids = P.tokens(root, 40)
    whole = P.oracle(root, w).feed(ids)
    for cut in (1, 2, 7):
        o = P.oracle(root, w)
        got = np.concatenate([o.feed(ids[i:i + cut]) for i in range(0, 40, cut)])
        assert np.abs(got - whole).max() < 1e-9


def test_oracle_convolution_is_numpys():
    from oracle import pomelix as O
    rng = np.random.default_rng(0)
    u, w = rng.standard_normal((12, 3)), rng.standard_normal((3, 4))
    got = O.short_convolution(u, w, np.zeros((3, 3)))
    for c in range(3):
        assert np.allclose(got[:, c], np.convolve(u[:, c], w[c, ::-1])[:12])
    past = rng.standard_normal((3, 3))
    both = O.short_convolution(np.concatenate([past, u]), w, np.zeros((3, 3)))
    assert np.allclose(O.short_convolution(u, w, past), both[3:])


def test_oracle_attention_is_causal_and_grouped():
    from oracle import pomelix as O
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((5, 4, 6)), rng.standard_normal((8, 2, 6)), rng.standard_normal((8, 2, 3))
    got = O.grouped_attention(q, k, v, 3, 0.7)
    s = np.einsum("ihd,jhd->hij", q, k.repeat(2, axis=1)) * 0.7
    s = np.where(np.arange(8)[None, None, :] <= (3 + np.arange(5))[None, :, None], s, -np.inf)
    a = np.exp(s) / np.exp(s).sum(-1, keepdims=True)
    assert np.allclose(got, np.einsum("hij,jhe->ihe", a, v.repeat(2, axis=1)))


def test_oracle_temperature_steps():
    from oracle import pomelix as O
    t = [O.query_temperature(p, 2.0, 5) for p in range(11)]
    assert t[:4] == [1.0] * 4 and t[4] == t[8] == 1 + 2 * np.log(2) and t[9] == t[10] == 1 + 2 * np.log(3)


def test_oracle_mixing_begins_at_the_first_layer_that_mixes():
    """The first mixing layer's own share changes nothing, a later one's does."""
    root = P.model([P.layer(P.mixer(v_mix=False)), P.layer(), P.layer()])
    w = P.weights(root)
    ids = P.tokens(root, 10)
    want = P.oracle(root, w).feed(ids)
    other = dict(w, **{"l1.mix.vmix": P.to_bf16(np.float32(0.9)).reshape(())})
    assert np.array_equal(P.oracle(root, other).feed(ids), want)
    other = dict(w, **{"l2.mix.vmix": P.to_bf16(np.float32(0.9)).reshape(())})
    assert np.abs(P.oracle(root, other).feed(ids) - want).max() > 1e-3
