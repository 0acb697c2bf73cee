"""Layered decoders on the GPU against the plain restatement: each mechanism alone, portions of prompts, decoding, reused
pages, unusual sizes, both precisions, and greedy generation through the worker."""
import io
import json

import numpy as np
import pytest

from tests import layered_models as L

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def run(root, w, ids, dtype, cuts=None, context=None):
    """Logits of every row, the prompt cut into portions of the given sizes."""
    m = L.engine(root, w, context or len(ids) + 8, dtype)
    try:
        return feed(m, ids, cuts)
    finally:
        m.close()


def feed(m, ids, cuts=None):
    out, at = [], 0
    for n in cuts or [len(ids)]:
        part = ids[at:at + n]
        if len(part):
            out.append(m.prefill_rows(part, range(len(part))))
        at += n
    assert at >= len(ids)
    return np.concatenate(out)


def close(got, want, dtype, factor=1.0):
    e = L.error(got, want)
    assert e.max() <= factor * L.LIMIT[dtype], (int(e.argmax()), float(e.max()))


@BOTH
def test_embedding_bigram_and_last_norm(dtype):
    """norm1 = -1 makes the only sublayer add exactly nothing."""
    root = L.model([L.layer(ff=None)], mul_prev=4099, mul_cur=977, buckets=11)
    w = L.weights(root, norm1=-1.0)
    ids = L.tokens(root, 70)
    ids[5:9] = ids[4]
    want = L.oracle(root, w).feed(ids)
    close(run(root, w, ids, dtype), want, dtype)
    close(run(root, w, ids, dtype, [1] * 70), want, dtype)
    close(run(root, w, ids, dtype, [2] * 35), want, dtype)


@BOTH
@pytest.mark.parametrize("mix", [
    dict(), dict(heads=1, dim=64, rot_dim=64, vdim=64, kv_rank=64), dict(heads=5, dim=7, rot_dim=2, vdim=3, kv_rank=5),
    dict(heads=3, dim=70, rot_dim=36, vdim=130, kv_rank=100, dims=20), dict(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512),
    dict(heads=2, dim=192, rot_dim=64, vdim=256, kv_rank=320), dict(heads=2, dim=260, rot_dim=32, vdim=40, kv_rank=48),
    dict(heads=20, dim=32, rot_dim=16, vdim=48, kv_rank=130)])
@pytest.mark.parametrize("scaling", [None, L.YARN])
def test_attention_alone(dtype, mix, scaling):
    root = L.model([L.layer(L.mixer(scaling=scaling, **mix), ff=None)])
    root["layers"][0]["mixer"]["scale"] = 2.0 / np.sqrt(root["layers"][0]["mixer"]["dim"])
    w = L.weights(root, seed=2)
    ids = L.tokens(root, 150)
    want = L.oracle(root, w).feed(ids)
    close(run(root, w, ids, dtype), want, dtype)
    close(run(root, w, ids, dtype, [100, 20, 3, 2] + [1] * 25), want, dtype)


@BOTH
@pytest.mark.parametrize("ff,limit", [(40, 0.7), (16, 3.0), (1, 1.0), (200, 0.25)])
def test_feed_forward_alone(dtype, ff, limit):
    root = L.model([L.layer(ff=ff, limit=limit)])
    w = L.weights(root, seed=3, norm1=-1.0)
    ids = L.tokens(root, 40)
    want = L.oracle(root, w).feed(ids)
    close(run(root, w, ids, dtype), want, dtype)
    close(run(root, w, ids, dtype, [20] + [1] * 20), want, dtype)


@pytest.mark.parametrize("scaling", [dict(factor=8.0, original=64, fast=32.0, slow=1.0), dict(factor=2.0, original=4000, fast=4.0, slow=3.9),
                                     dict(factor=1.0, original=128, fast=2.0, slow=0.5), dict(factor=40.0, original=7, fast=64.0, slow=32.0)])
def test_rotation_ramps(scaling):
    """Ramps that are clamped at either end, empty, or collapsed onto one pair."""
    root = L.model([L.layer(L.mixer(rot_dim=24, dim=8, scale=1.0, base=300.0, scaling=scaling), ff=None)])
    w = L.weights(root, seed=4)
    ids = L.tokens(root, 90)
    close(run(root, w, ids, "float32"), L.oracle(root, w).feed(ids), "float32")


def deep(**kw):
    return L.model([L.layer(), L.layer(L.mixer(heads=3, scaling=L.YARN, vdim=36, kv_rank=40), ff=56, limit=1.0), L.layer(ff=None),
                    L.layer(weights_of=0), L.layer(L.mixer(heads=3, scaling=L.YARN, vdim=36, kv_rank=40), ff=56, limit=1.0, weights_of=1)],
                   **kw)


@BOTH
def test_whole_model_prompt_portions_and_decoding(dtype):
    root = deep()
    w = L.weights(root, seed=5)
    ids = L.tokens(root, 200)
    want = L.oracle(root, w).feed(ids)
    m = L.engine(root, w, 256, dtype)
    first = feed(m, ids)
    close(first, want, dtype)
    for cuts in ([2] * 100, [64, 64, 64, 8], [63, 2, 63, 72], [17, 16, 3, 37, 2, 65, 60], [150] + [1] * 50, [1] * 200):
        m.reset()
        close(feed(m, ids, cuts), want, dtype)
    m.reset()
    again = feed(m, ids)
    assert np.array_equal(again, first)      # the cache's pages were used by other runs in between
    m.close()


@BOTH
def test_pages_used_again_by_other_sequences(dtype):
    root = deep()
    w = L.weights(root, seed=6)
    m = L.engine(root, w, 192, dtype)
    for seed, n in ((1, 190), (2, 5), (3, 129), (4, 64), (5, 1)):
        ids = L.tokens(root, n, seed=seed)
        m.reset()
        cut = max(1, n // 3)
        close(feed(m, ids, [cut, n - cut] if n > 1 else None), L.oracle(root, w).feed(ids), dtype)
    m.close()


@BOTH
def test_rewind_keeps_the_previous_token(dtype):
    """Rewinding to a position and feeding other tokens: the bigram of the first new row needs the token before it."""
    root = deep()
    w = L.weights(root, seed=7)
    a, b = L.tokens(root, 100, seed=1), L.tokens(root, 60, seed=2)
    m = L.engine(root, w, 192, dtype)
    feed(m, a)
    m.rewind(70)
    want = L.oracle(root, w).feed(np.concatenate([a[:70], b]))[70:]
    close(feed(m, b, [1, 2, 57]), want, dtype)
    m.rewind(0)
    close(feed(m, b), L.oracle(root, w).feed(b), dtype)
    m.close()


@BOTH
def test_far_keys_at_page_borders(dtype):
    """One cached row outshines all others for every later query: a marker token whose latent only matches the query
    everybody asks.  Dropping, doubling or shifting that row would change every logit."""
    # width 64: entry 0 of the embedding marks the needle, entry 1 is in every token
    mix = L.mixer(heads=1, dim=16, rot_dim=2, vdim=16, kv_rank=16, scale=1.0, base=1e6)
    root = L.model([L.layer(mix, ff=None)], width=64, vocab=40, scale=1.0)
    w = {k: L.from_bf16(v).copy() for k, v in L.weights(root, seed=8, norm1=0.0).items()}
    rng = np.random.default_rng(9)
    w["embed"] = 0.3 * rng.standard_normal((40, 64)).astype(np.float32)
    w["embed"][:, 0], w["embed"][:, 1] = 0.0, 2.0
    w["embed"][39, 0], w["embed"][39, 1] = 8.0, 0.0
    w["bigram"][:] *= 0.05
    w["bigram"][:, 0] = 0.0
    w["l0.mix.q"][:] = 0.0
    w["l0.mix.q"][0, 1] = 5.0                         # everybody asks for latent entry 0
    w["l0.mix.dkv"][0, :] = 0.0
    w["l0.mix.dkv"][0, 0] = 6.0                       # the needle alone has it
    w["l0.mix.uk"][:] = 0.0
    w["l0.mix.uk"][0, 0] = 1.0
    w = {k: L.to_bf16(v) for k, v in w.items()}
    n = 330
    for needle in (0, 1, 62, 63, 64, 65, 127, 128, 255, 256, 319):
        ids = L.tokens(root, n, seed=needle) % 39
        ids[needle] = 39
        want = L.oracle(root, w).feed(ids)
        gone = ids.copy()
        gone[needle] = 3
        assert L.error(L.oracle(root, w).feed(gone)[-1:], want[-1:]).max() > 0.3     # the row does decide
        m = L.engine(root, w, n, dtype)
        close(feed(m, ids), want, dtype)
        m.reset()
        close(feed(m, ids, [300] + [1] * 30), want, dtype)
        m.reset()
        close(feed(m, ids, [128, 64, 2, 64, 7, 65]), want, dtype)
        m.close()


@BOTH
def test_long_decoding(dtype):
    root = deep(vocab=130, width=128)
    w = L.weights(root, seed=10)
    ids = L.tokens(root, 700)
    want = L.oracle(root, w).feed(ids)
    m = L.engine(root, w, 700, dtype)
    m.prefill(ids[:20])
    got = np.stack([m.step(int(t)) for t in ids[20:]])
    close(got, want[20:], dtype)
    m.close()


@BOTH
def test_several_passes_of_rows(dtype):
    """A prompt longer than one pass (4 096 rows), portions around it."""
    root = L.model([L.layer(L.mixer(heads=1, scaling=L.YARN), ff=None), L.layer(L.mixer(heads=2), ff=24)])
    w = L.weights(root, seed=11)
    n = 4300 if dtype == "bfloat16" else 4110
    ids = L.tokens(root, n)
    wanted = [0, 1, 63, 64, 4094, 4095, 4096, 4097, n - 1]
    want = L.oracle(root, w).feed(ids)[wanted]
    m = L.engine(root, w, n, dtype)
    close(m.prefill_rows(ids, wanted), want, dtype)
    m.close()


@pytest.mark.parametrize("sizes", [dict(vocab=3, width=8), dict(vocab=1000, width=200), dict(vocab=257, width=1030)])
def test_other_model_sizes(sizes):
    root = deep(**sizes)
    w = L.weights(root, seed=12)
    ids = L.tokens(root, 90)
    want = L.oracle(root, w).feed(ids)
    for dtype in ("float32", "bfloat16"):
        close(run(root, w, ids, dtype, [70] + [1] * 20), want, dtype)


def test_precisions_differ_and_residual_is_f32():
    """A residual stream rounded to bf16 after each of many layers would exceed the bf16 bar that a f32 one keeps."""
    root = L.model([L.layer(L.mixer(heads=2))] + [L.layer(L.mixer(heads=2), weights_of=0) for _ in range(23)])
    w = L.weights(root, seed=13, norm1=-0.75, norm2=-0.75)
    ids = L.tokens(root, 60)
    want = L.oracle(root, w).feed(ids)
    close(run(root, w, ids, "float32"), want, "float32", 2.0)
    close(run(root, w, ids, "bfloat16", [30] + [1] * 30), want, "bfloat16")


def test_read_outs_and_sampling():
    root = deep()
    w = L.weights(root, seed=14)
    ids = L.tokens(root, 50)
    m = L.engine(root, w, 128, "float32")
    m.prefill(ids)
    want = L.oracle(root, w).feed(ids)[-1]
    close(m.logits()[None], want[None], "float32")
    assert m.argmax() == int(want.argmax())
    lp = m.log_probabilities()
    assert np.allclose(lp, want - np.log(np.exp(want - want.max()).sum()) - want.max(), atol=1e-3)
    assert m.sample() == int(want.argmax())
    assert {m.sample(seed=s, temperature=1.0, top_k=3) for s in range(40)} <= set(np.argsort(want)[-3:].tolist())
    info = m.info()
    assert info.position == 50 and info.vocab_size == root["vocab"] and info.weight_bytes > 0 and info.kv_bytes_per_token > 0
    m.close()


def test_library_loader_serves_the_same_model(tmp_path):
    from stark_b200.artifact import write_layered
    from stark_b200.engine import LayeredModel
    root = deep()
    w = L.weights(root, seed=21)
    write_layered(tmp_path, root, w)
    ids = L.tokens(root, 90)
    a, b = LayeredModel.from_artifact(tmp_path, 128), LayeredModel.load_path(tmp_path, 128)
    assert np.array_equal(feed(a, ids, [40, 50]), feed(b, ids, [40, 50]))
    a.close()
    b.close()


def greedy_reference(root, w, ids, n):
    o = L.oracle(root, w)
    row = o.feed(ids)[-1]
    out = []
    for _ in range(n):
        out.append(int(row.argmax()))
        row = o.feed([out[-1]])[-1]
    return out


def test_device_chained_greedy():
    root = deep()
    w = L.weights(root, seed=15)
    ids = L.tokens(root, 30)
    m = L.engine(root, w, 128, "float32")
    m.prefill(ids)
    assert m.generate_greedy(40).tolist() == greedy_reference(root, w, ids, 41)
    m.close()


def test_generation_through_the_worker(tmp_path, monkeypatch):
    """The worker's own request path: prompt, greedy tokens, prefix reuse on the second request."""
    from stark_b200 import worker as W
    from stark_b200.artifact import write_layered
    root = deep(vocab=90)
    w = L.weights(root, seed=16)
    write_layered(tmp_path, root, w)
    monkeypatch.setenv("STARK_B200_WORKER_DTYPE", "float32")
    monkeypatch.setenv("STARK_B200_WORKER_CONTEXT", "2304")
    backend = W.B200Backend(tmp_path)
    worker = W.GenerationWorker(backend, W.Budget(64), True)
    prompt = L.tokens(root, 1500).tolist()
    want = greedy_reference(root, w, prompt, 12)
    for tail in ([], [5, 6]):
        request = {"operation": "generate", "input_token_ids": prompt + tail, "context_tokens": 2200, "max_new_tokens": 12,
                   "cache_scope": "ab" * 16}
        reply = worker.handle(dict(request), io.BytesIO())
        assert reply["generated_token_ids"] == (want if not tail else greedy_reference(root, w, prompt + tail, 12)), json.dumps(reply)[:300]
    plan = worker.handle({"operation": "plan_generation", "input_tokens": 100, "context_tokens": 2000}, io.BytesIO())
    assert plan["context_tokens"] == 2000
    logits, _ = backend.score(prompt[:40])
    close(logits[None], L.oracle(root, w).feed(prompt[:40])[-1:], "float32")
    backend.model.close()


def test_dense_prefill_rows_agrees_with_steps():
    """The row read-out on a family without a several-rows form: the portion is cut behind each wanted row."""
    from stark_b200 import synthetic as S
    from stark_b200.engine import DenseModel
    cfg = S.CONFIGS["tiny"]
    m = DenseModel.load(cfg, S.dense_weights(cfg, seed=3, zero_point=7.5), context_tokens=128)
    ids = S.prompt(cfg, 60, seed=17)
    rows = m.prefill_rows(ids, [0, 20, 59])
    m.reset()
    steps = [m.step(int(t)) for t in ids]
    for got, at in zip(rows, (0, 20, 59)):
        assert L.error(got, steps[at].astype(np.float64)) < 0.05
    m.close()


def test_invalid_requests_are_refused_on_the_host():
    from stark_b200._lib import StarkB200Error
    root = deep()
    m = L.engine(root, L.weights(root), 64, "bfloat16")
    for ids, rows in ((L.tokens(root, 65), []), ([root["vocab"]], [0]), ([1, 2], [2]), ([1, 2, 3], [1, 1])):
        with pytest.raises(StarkB200Error):
            m.prefill_rows(ids, rows)
    m.reset()
    assert m.position == 0
    m.close()
