"""Pomelix on the GPU against the plain restatement: each mechanism alone, portions of prompts, decoding, reused pages,
rewinds, unusual sizes, both precisions, and greedy generation through the worker."""
import io
import json

import numpy as np
import pytest

from tests import pomelix_models as P
from tests.test_layered_gpu import close, feed

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def check(root, w, ids, dtype, cuts=(None,), context=None, factor=1.0):
    """One model, the prompt fed once per way of cutting it."""
    want = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, context or len(ids) + 8, dtype)
    try:
        for c in cuts:
            m.reset()
            close(feed(m, ids, c), want, dtype, factor)
    finally:
        m.close()
    return want


def edited(w, **tensors):
    """Tensors replaced, names with dots as double underscores."""
    return dict(w, **{k.replace("__", "."): P.to_bf16(np.asarray(v, np.float32)).reshape(np.shape(v)) for k, v in tensors.items()})


@BOTH
def test_embedding_and_tied_read_out(dtype):
    """Layer scales of zero leave the embedding under the last norm."""
    root = P.model([P.layer(), P.layer(ff=None)])
    ids = P.tokens(root, 70)
    check(root, P.weights(root, ls1=0.0, ls2=0.0), ids, dtype, (None, [1] * 70, [2] * 35))


@BOTH
@pytest.mark.parametrize("mult,ls1,ls2", [(1.0, 1.0, 0.0), (-0.35, 0.0, 2.5), (0.25, -1.5, 3.0)])
def test_residual_and_layer_scales(dtype, mult, ls1, ls2):
    root = P.model([P.layer(), P.layer(ff=90), P.layer(ff=None)], residual_mult=mult)
    ramp = np.linspace(0.5, 1.5, root["width"])
    w = P.weights(root, seed=1, ls1=ls1 * ramp, ls2=ls2 * ramp[::-1])
    check(root, w, P.tokens(root, 60), dtype, (None, [30] + [1] * 30))


@BOTH
@pytest.mark.parametrize("ff", [1, 16, 40, 200])
def test_feed_forward_alone(dtype, ff):
    root = P.model([P.layer(ff=ff)])
    w = P.weights(root, seed=2, ls1=0.0)
    check(root, w, P.tokens(root, 40), dtype, (None, [20] + [1] * 20))


@BOTH
@pytest.mark.parametrize("mix", [
    dict(), dict(heads=1, kv_heads=1, dim=64, vdim=64), dict(heads=5, kv_heads=1, dim=7, vdim=3), dict(heads=3, kv_heads=3, dim=70, vdim=130),
    dict(heads=8, kv_heads=2, dim=128, vdim=128), dict(heads=20, kv_heads=1, dim=16, vdim=40), dict(heads=36, kv_heads=2, dim=24, vdim=66),
    dict(heads=2, kv_heads=1, dim=192, vdim=256), dict(heads=2, kv_heads=1, dim=256, vdim=1), dict(heads=2, kv_heads=2, dim=300, vdim=20),
    dict(heads=4, kv_heads=2, dim=20, vdim=500), dict(heads=2, kv_heads=1, dim=1, vdim=17)])
def test_attention_sizes(dtype, mix):
    root = P.model([P.layer(P.mixer(**mix), ff=None)])
    m = root["layers"][0]["mixer"]
    m["scale"] = 2.0 / np.sqrt(m["dim"])
    w = P.weights(root, seed=3)
    check(root, w, P.tokens(root, 150), dtype, (None, [100, 20, 3, 2] + [1] * 25))


@BOTH
@pytest.mark.parametrize("scale,coef,every", [(1.5, 0.0, 1), (0.02, 3.0, 7), (1.2, 0.8, 64), (0.3, -0.9, 10), (-0.4, 0.5, 33)])
def test_scales_and_temperatures(dtype, scale, coef, every):
    """Large scales leave the range in which a bound stands in for the maximum; a negative coefficient turns the queries
    around; a negative scale turns the scores."""
    root = P.model([P.layer(P.mixer(heads=2, kv_heads=1, dim=48, scale=scale, coef=coef, every=every), ff=None)])
    w = P.weights(root, seed=4)
    check(root, w, P.tokens(root, 180), dtype, (None, [130] + [1] * 50, [2] * 90), factor=1.0 if dtype == "float32" else 1.5)


@pytest.mark.parametrize("every", [1, 7, 64])
def test_temperature_steps_where_it_should(every):
    """Every row of the prompt with its own temperature: a step one position early or late shows in that row."""
    root = P.model([P.layer(P.mixer(heads=2, kv_heads=1, dim=16, scale=0.5, coef=2.0, every=every), ff=None)])
    w = P.weights(root, seed=5, conv=[0.0, 0.0, 0.0, 1.0])
    ids = P.tokens(root, 140)
    want = check(root, w, ids, "float32", (None, [1] * 140, [63, 2, 63, 12]))
    late = dict(root["layers"][0]["mixer"], q_temp={"coef": 2.0, "every": every + 1})
    other = P.oracle(P.model([P.layer(late, ff=None)]), w).feed(ids)
    assert P.error(other, want).max() > 0.01


@BOTH
@pytest.mark.parametrize("taps", [1, 2, 3, 5, 17, 33])
def test_convolutions(dtype, taps):
    """All weight on the oldest tap: each row depends on the projected row taps - 1 positions back and on no other, so a
    shifted, lost or stale row of the state changes everything behind it."""
    root = P.model([P.layer(P.mixer(conv=taps), ff=None), P.layer(P.mixer(conv=taps, heads=2, kv_heads=1, vdim=56))])
    oldest = np.zeros(taps)
    oldest[0], oldest[-1] = 1.0, 1.0 if taps == 1 else 0.02
    w = P.weights(root, seed=6, conv=oldest)
    check(root, w, P.tokens(root, 170), dtype,
          (None, [1] * 170, [2] * 85, [3, 2, 100, 16, 17, 2, 30], [63, 2, 62, 2, 41], [130] + [1] * 40))


@BOTH
def test_layers_without_convolution_or_temperature(dtype):
    root = P.model([P.layer(), P.layer(P.mixer(conv=3)), P.layer()])
    w = P.weights(root, seed=7, l1_mix_q_conv=[0.0, 0.0, 1.0], l1_mix_k_conv=[0.0, 0.0, 1.0], l1_mix_v_conv=[0.0, 0.0, 1.0])
    root["layers"][1]["mixer"]["q_temp"]["coef"] = 0.0
    ids = P.tokens(root, 90)
    want = P.oracle(root, w).feed(ids)
    m = root["layers"][1]["mixer"]
    m["conv"] = m["q_temp"] = None
    eng = P.engine(root, {k: v for k, v in w.items() if not (k.startswith("l1") and k.endswith("conv"))}, 96, dtype)
    close(feed(eng, ids, [60, 5] + [1] * 25), want, dtype)
    eng.close()


@BOTH
def test_value_mixing(dtype):
    """Shares of one (a later layer's values are the first mixing layer's), of zero, and layers that do not mix between
    and before."""
    plain = P.mixer(v_mix=False, dim=30, vdim=44, heads=4)
    root = P.model([P.layer(plain, ff=None), P.layer(), P.layer(plain), P.layer(P.mixer(dim=50)), P.layer()])
    w = edited(P.weights(root, seed=8), l1__mix__vmix=0.77, l3__mix__vmix=1.0, l4__mix__vmix=0.0)
    check(root, w, P.tokens(root, 130), dtype, (None, [1] * 130, [70, 2, 58]))
    w = edited(w, l4__mix__vmix=-0.5)
    check(root, w, P.tokens(root, 80), dtype, (None, [40] + [1] * 40))


def deep(**kw):
    return P.model([P.layer(), P.layer(P.mixer(heads=4, kv_heads=1, dim=70, conv=2, v_mix=False), ff=None),
                    P.layer(P.mixer(heads=2, kv_heads=2, dim=130, conv=3, every=5, scale=0.1), ff=100), P.layer(ff=24)], **kw)


@BOTH
def test_whole_model_prompt_portions_and_decoding(dtype):
    root = deep()
    w = P.weights(root, seed=9)
    ids = P.tokens(root, 200)
    want = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, 256, dtype)
    first = feed(m, ids)
    close(first, want, dtype)
    for cuts in ([2] * 100, [64, 64, 64, 8], [63, 2, 63, 72], [17, 16, 3, 37, 2, 65, 60], [150] + [1] * 50, [1] * 200):
        m.reset()
        close(feed(m, ids, cuts), want, dtype)
    m.reset()
    assert np.array_equal(feed(m, ids), first)      # the pages and the convolutions' state were used by other runs between
    m.close()


def test_residual_streams_layer_by_layer():
    """The oracle's stream behind every layer, through models cut off there."""
    root = deep()
    w = P.weights(root, seed=10)
    ids = P.tokens(root, 40)
    for n in range(1, len(root["layers"]) + 1):
        part = dict(root, layers=root["layers"][:n])
        check(part, {k: v for k, v in w.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}, ids, "float32")


@BOTH
def test_pages_used_again_by_other_sequences(dtype):
    root = deep()
    w = P.weights(root, seed=11)
    m = P.engine(root, w, 192, dtype)
    for seed, n in ((1, 190), (2, 5), (3, 129), (4, 64), (5, 1), (6, 2), (7, 66)):
        ids = P.tokens(root, n, seed=seed)
        m.reset()
        cut = max(1, n // 3)
        close(feed(m, ids, [cut, n - cut] if n > 1 else None), P.oracle(root, w).feed(ids), dtype)
    m.close()


@BOTH
def test_rewind_restores_the_convolutions(dtype):
    root = deep()
    root["layers"][0]["mixer"]["conv"] = 9
    w = P.weights(root, seed=12)
    a = P.tokens(root, 180, seed=1)
    m = P.engine(root, w, 256, dtype)
    feed(m, a, [100, 50] + [1] * 30)
    for n, (to, cuts) in enumerate(((179, [1, 2, 20]), (130, [2, 21]), (128, [1] * 23), (127, [23]), (70, [1, 2, 20]), (64, [2, 21]),
                                    (65, [23]), (63, [23]), (3, [5, 18]), (1, [23]), (0, [23]))):
        b = P.tokens(root, 23, seed=20 + n)
        m.rewind(to)
        assert m.position == to
        a = np.concatenate([a[:to], b])
        close(feed(m, b, cuts), P.oracle(root, w).feed(a)[to:], dtype)
    m.close()


@pytest.mark.parametrize("settings", [dict(grouped_cluster=1), dict(grouped_cluster=2, grouped_splits=3), dict(grouped_cluster=8),
                                      dict(grouped_cluster=4, grouped_splits=9), dict(pdl=0)])
def test_spans_of_the_decode_attention(settings):
    """Recorded anew in the middle of a sequence with other divisions of the cache: more spans than pages, one span."""
    root = P.model([P.layer(P.mixer(heads=3, kv_heads=1, conv=5)), P.layer(P.mixer(heads=20, kv_heads=1, dim=64))])
    w = P.weights(root, seed=13)
    ids = P.tokens(root, 420)
    want = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, 448, "bfloat16")
    try:
        close(feed(m, ids[:300], [290] + [1] * 10), want[:300], "bfloat16")
        m.recapture(**settings)
        close(feed(m, ids[300:], [1] * 60 + [2, 30] + [1] * 28), want[300:], "bfloat16")
        m.reset()
        close(feed(m, ids[:140], [1] * 140), want[:140], "bfloat16")
    finally:
        m.recapture(**{k: 1 if k == "pdl" else 0 for k in settings})
        m.close()


@pytest.mark.parametrize("dim,vdim", [(16, 16), (128, 128), (180, 70), (250, 250)])
def test_spans_longer_than_the_pages_in_flight(dim, vdim):
    """One CTA reads the whole cache: pages take the places of pages already read, whatever number of them fits."""
    root = P.model([P.layer(P.mixer(heads=5, kv_heads=1, dim=dim, vdim=vdim, scale=1.0 / np.sqrt(dim)), ff=None)])
    w = P.weights(root, seed=25)
    ids = P.tokens(root, 900)
    want = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, 900, "bfloat16")
    try:
        m.recapture(grouped_cluster=1, grouped_splits=1)
        for at in (60, 190, 250, 330, 640, 885):
            m.reset()
            m.prefill(ids[:at])
            close(feed(m, ids[at:at + 12], [1] * 12), want[at:at + 12], "bfloat16")
    finally:
        m.recapture(grouped_cluster=0, grouped_splits=0)
        m.close()


def needle_model(scale=0.75, coef=0.3, every=16):
    """Every query asks for one direction, which only the needle token's key has: entry 0 of the embedding marks the needle,
    entry 1 is in every other token."""
    root = P.model([P.layer(P.mixer(heads=2, kv_heads=1, dim=16, vdim=16, conv=3, scale=scale, coef=coef, every=every, v_mix=False),
                            ff=None)], width=64, vocab=40, residual_mult=1.0)
    w = {k: P.from_bf16(v).copy() for k, v in P.weights(root, seed=14, norm1=1.0, ls1=1.0).items()}
    rng = np.random.default_rng(9)
    w["embed"] = 0.3 * rng.standard_normal((40, 64)).astype(np.float32)
    w["embed"][:, 0], w["embed"][:, 1] = 0.0, 2.0
    w["embed"][39, 0], w["embed"][39, 1] = 8.0, 0.0
    for name in ("q", "k"):
        w[f"l0.mix.{name}"][:] = 0.0
        w[f"l0.mix.{name}.conv"][:] = [0.0, 0.0, 1.0]
    w["l0.mix.q"][0, 0] = w["l0.mix.q"][16, 0] = w["l0.mix.q"][0, 1] = w["l0.mix.q"][16, 1] = 5.0
    w["l0.mix.k"][0, 0] = 6.0
    w["l0.mix.k"][1, 1] = 6.0
    w["l0.mix.v"] *= 3.0
    return root, {k: P.to_bf16(v).reshape(v.shape) for k, v in w.items()}


@BOTH
def test_far_keys_at_page_borders(dtype):
    """One cached row outshines all others for every later query.  Dropping, doubling or shifting it would change every
    logit."""
    root, w = needle_model()
    n = 330
    for needle in (0, 1, 15, 16, 62, 63, 64, 65, 127, 128, 191, 255, 256, 319):
        ids = P.tokens(root, n, seed=needle) % 39
        ids[needle] = 39
        want = P.oracle(root, w).feed(ids)
        gone = ids.copy()
        gone[needle] = 3
        assert P.error(P.oracle(root, w).feed(gone)[-1:], want[-1:]).max() > 0.3     # the row does decide
        m = P.engine(root, w, n, dtype)
        for cuts in (None, [300] + [1] * 30, [128, 64, 2, 64, 7, 65], [needle + 1, 2, n - needle - 3]):
            m.reset()
            close(feed(m, ids, cuts), want, dtype)
        m.close()


@BOTH
def test_first_tokens(dtype):
    """Sequences shorter than the convolutions reach, one token at a time and at once."""
    root = deep()
    root["layers"][0]["mixer"]["conv"] = 12
    w = P.weights(root, seed=15)
    m = P.engine(root, w, 64, dtype)
    for n in (1, 2, 3, 4, 13):
        ids = P.tokens(root, n, seed=n)
        want = P.oracle(root, w).feed(ids)
        for cuts in (None, [1] * n, [2] * ((n + 1) // 2)):
            m.reset()
            close(feed(m, ids, cuts), want, dtype)
    m.close()


@BOTH
def test_long_decoding(dtype):
    root = deep(vocab=130, width=128)
    w = P.weights(root, seed=16)
    ids = P.tokens(root, 700)
    want = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, 700, dtype)
    m.prefill(ids[:20])
    got = np.stack([m.step(int(t)) for t in ids[20:]])
    close(got, want[20:], dtype)
    m.close()


@BOTH
def test_several_passes_of_rows(dtype):
    """A prompt longer than one pass (4 096 rows), portions around it, then decoding with several clusters of spans."""
    root = P.model([P.layer(P.mixer(heads=1, kv_heads=1, conv=3), ff=None), P.layer(P.mixer(heads=2, kv_heads=1), ff=24)])
    w = P.weights(root, seed=17)
    n = 4300 if dtype == "bfloat16" else 4110
    ids = P.tokens(root, n)
    wanted = [0, 1, 63, 64, 4094, 4095, 4096, 4097, n - 1]
    full = P.oracle(root, w).feed(ids)
    m = P.engine(root, w, n, dtype)
    close(m.prefill_rows(ids, wanted), full[wanted], dtype)
    m.rewind(n - 9)
    close(feed(m, ids[n - 9:], [1] * 9), full[n - 9:], dtype)
    m.close()


@pytest.mark.parametrize("sizes", [dict(vocab=3, width=8), dict(vocab=1000, width=200), dict(vocab=257, width=1030)])
def test_other_model_sizes(sizes):
    root = deep(**sizes)
    w = P.weights(root, seed=18)
    ids = P.tokens(root, 90)
    for dtype in ("float32", "bfloat16"):
        check(root, w, ids, dtype, ([70] + [1] * 20,))


def test_residual_stream_is_f32():
    """A residual stream rounded to bf16 after each of many layers would exceed the bf16 bar that a f32 one keeps."""
    root = P.model([P.layer(P.mixer(heads=2)) for _ in range(24)], residual_mult=0.2)
    w = P.weights(root, seed=19)
    ids = P.tokens(root, 60)
    check(root, w, ids, "float32", factor=2.0)
    check(root, w, ids, "bfloat16", ([30] + [1] * 30,))


def test_read_outs_and_sampling():
    root = deep()
    w = P.weights(root, seed=20)
    ids = P.tokens(root, 50)
    m = P.engine(root, w, 128, "float32")
    m.prefill(ids)
    want = P.oracle(root, w).feed(ids)[-1]
    close(m.logits()[None], want[None], "float32")
    assert m.argmax() == int(want.argmax()) == m.sample()
    lp = m.log_probabilities()
    assert np.allclose(lp, want - np.log(np.exp(want - want.max()).sum()) - want.max(), atol=1e-3)
    assert {m.sample(seed=s, temperature=1.0, top_k=3) for s in range(40)} <= set(np.argsort(want)[-3:].tolist())
    info = m.info()
    assert info.position == 50 and info.vocab_size == root["vocab"] and info.weight_bytes > 0 and info.kv_bytes_per_token > 0
    m.close()


def test_library_loader_serves_the_same_model(tmp_path):
    from stark_b200.artifact import write_layered
    from stark_b200.engine import LayeredModel
    root = deep()
    w = P.weights(root, seed=21)
    write_layered(tmp_path, root, w)
    ids = P.tokens(root, 90)
    a, b = LayeredModel.from_artifact(tmp_path, 128), LayeredModel.load_path(tmp_path, 128)
    assert np.array_equal(feed(a, ids, [40, 50]), feed(b, ids, [40, 50]))
    a.close()
    b.close()


def test_trace_replay_serves_the_family(tmp_path):
    from stark_b200 import registry
    from stark_b200.artifact import write_layered
    from stark_b200.trace import Replay
    root = deep()
    w = P.weights(root, seed=22)
    write_layered(tmp_path, root, w)
    m = registry.open_model(tmp_path).load(80, "float32")
    r = Replay(m)
    for name, n in (("a", 70), ("b", 9)):
        ids = P.tokens(root, n, seed=n)
        want = P.oracle(root, w).feed(ids)
        r.step({"step": 0, "entries": [{"id": name, "tokens": ids[:n - 3].tolist(), "want": []}]})
        got = r.step({"step": 1, "entries": [{"id": name, "tokens": ids[n - 3:].tolist(), "want": [2, 0]}], "end": [name]})
        close(np.frombuffer(got, "<f4").reshape(2, -1), want[[n - 1, n - 3]], "float32")
    m.close()


def greedy_reference(root, w, ids, n):
    o = P.oracle(root, w)
    row = o.feed(ids)[-1]
    out = []
    for _ in range(n):
        out.append(int(row.argmax()))
        row = o.feed([out[-1]])[-1]
    return out


def test_device_chained_greedy():
    root = deep()
    w = P.weights(root, seed=23)
    ids = P.tokens(root, 30)
    m = P.engine(root, w, 128, "float32")
    m.prefill(ids)
    assert m.generate_greedy(60).tolist() == greedy_reference(root, w, ids, 61)
    m.close()


def test_generation_through_the_worker(tmp_path, monkeypatch):
    """The worker's own request path: prompt, greedy tokens, prefix reuse on the second request."""
    from stark_b200 import worker as W
    from stark_b200.artifact import write_layered
    root = deep(vocab=90)
    w = P.weights(root, seed=24)
    write_layered(tmp_path, root, w)
    monkeypatch.setenv("STARK_B200_WORKER_DTYPE", "float32")
    monkeypatch.setenv("STARK_B200_WORKER_CONTEXT", "2304")
    backend = W.B200Backend(tmp_path)
    worker = W.GenerationWorker(backend, W.Budget(64), True)
    prompt = P.tokens(root, 1500).tolist()
    for tail in ([], [5, 6]):
        request = {"operation": "generate", "input_token_ids": prompt + tail, "context_tokens": 2200, "max_new_tokens": 12,
                   "cache_scope": "ab" * 16}
        reply = worker.handle(dict(request), io.BytesIO())
        assert reply["generated_token_ids"] == greedy_reference(root, w, prompt + tail, 12), json.dumps(reply)[:300]
    logits, _ = backend.score(prompt[:40])
    close(logits[None], P.oracle(root, w).feed(prompt[:40])[-1:], "float32")
    backend.model.close()


def test_configurations_the_engine_refuses():
    from stark_b200._lib import StarkB200Error
    bad = [P.model([P.layer(), P.layer(P.mixer(vdim=29))]),              # mixed values of different widths
           P.model([P.layer(P.mixer(conv=65))]), P.model([P.layer(P.mixer(dim=513))])]
    for root in bad:
        with pytest.raises(StarkB200Error):
            P.engine(root, P.weights(root), 64, "bfloat16")
