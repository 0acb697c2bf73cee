// The layered family: decoders whose configuration lists every layer's mixer and feed-forward (Guvulorn: latent
// attention, clamped gated feed-forwards, norms on the sublayers' outputs, a hashed bigram table beside the embedding,
// layers that use another layer's tensors).  This file holds what such a model owns -- tensors in the padded layout of
// layered.cuh, one latent cache per layer over the session's page table, the token history -- and what one token and one
// pass of prompt rows launch; stepping, recording, prompt loop, read-out, sampling and rewind are the shared token loop's.
//
// Per layer a token is seven launches (five without a feed-forward):
//   [queries | latent, key part] = W x    matvec; the residual add of the sublayer before it in the prologue
//   query, attend, value                  latent attention (latent_attention.cu)
//   y = W_o attn                          matvec
//   act = gate(W_gu x)                    matvec, x = x + norm1(y) in the prologue, biases and gate in the epilogue
//   y = W_down act                        matvec
// and the read-out matvec forms x + norm2(y) and the last norm in its prologue and the greedy pick in its epilogue.
#include "layered.cuh"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <new>

#include "model.cuh"
#include "prefill.cuh"
#include "tunables.cuh"

#define SB_TRY(expr)                        \
    do {                                    \
        stark_b200_status _s = (expr);      \
        if (_s != STARK_B200_OK) return _s; \
    } while (0)

namespace sb {

namespace {

struct LayerTensors {
    MatrixB16 qd, uk_uv, o, gate_up, down;
    float *latent_norm = nullptr, *norm1 = nullptr, *norm2 = nullptr, *gate_up_b = nullptr, *down_b = nullptr;
    uint32_t seen = 0;  // bit per tensor id
};
struct Layer {
    stark_b200_layer_desc d{};
    LatentShape s{};
    Rotation rot{};
    float *freq = nullptr;
    uint32_t ff_p = 0;
    uint32_t tensors = 0;  // index of the layer that holds them
    LayerTensors own;
    void *cache = nullptr;
};

constexpr uint32_t kAttendRows = 64;    // rows of a pass the absorbed attention takes at a time
constexpr uint32_t kReadoutRows = 128;  // rows read out at a time

}  // namespace

struct LayeredState {
    stark_b200_layered_config c{};
    std::vector<Layer> layers;
    uint32_t width_p = 0;
    bool f32 = false;
    uint16_t *embed = nullptr, *bigram = nullptr;
    MatrixB16 head;
    float *embed_norm = nullptr, *final_norm = nullptr;
    uint32_t seen = 0;
    uint32_t *history = nullptr;  // token ids by position: where a row's previous token comes from
    // widest rows over the layers
    uint32_t max_qd = 0, max_attn = 0, max_ff = 0, max_expand = 0;
    size_t query_floats = 0, partial_floats = 0;
    // one token
    float *x[2] = {nullptr, nullptr}, *y = nullptr, *qd = nullptr, *attn = nullptr, *act = nullptr;
    float *queries = nullptr, *partials = nullptr;
    // a pass of rows
    uint32_t rows = 0;
    float *rx = nullptr, *ry = nullptr;
    uint16_t *rx_b16 = nullptr;
    void *rqd = nullptr, *rattn = nullptr, *ract = nullptr;  // bf16, or f32 in the 32-bit form
    float *rgu = nullptr;                                    // 32-bit form only
    uint16_t *expanded = nullptr;
    size_t expanded_rows = 0;
    uint32_t *picked = nullptr;
    void *picked_x = nullptr;
    float *picked_logits = nullptr;
};

namespace {

// Row r of a fused gate / up pair: 16 gate rows, 16 up rows in turn (a tile of the contraction holds both halves).
uint32_t pair_row(uint32_t r, bool up) { return (r / 16u) * 32u + (up ? 16u : 0u) + r % 16u; }

stark_b200_status alloc_matrix(MatrixB16 &m, uint32_t rows, uint32_t cols) {
    if (m.data) return STARK_B200_OK;
    SB_TRY(dmalloc(&m.data, (size_t)rows * cols));
    m.rows = rows;
    m.cols = cols;
    SB_CUDA(cudaMemset(m.data, 0, m.bytes()));
    return STARK_B200_OK;
}

// Rows [src_row, src_row + rows) x columns [src_col, src_col + cols) of a host matrix into the padded device matrix.
stark_b200_status place(MatrixB16 &m, uint32_t row, uint32_t col, const uint16_t *src, uint32_t src_ld, uint32_t src_row,
                        uint32_t src_col, uint32_t rows, uint32_t cols) {
    SB_CUDA(cudaMemcpy2D(m.data + (size_t)row * m.cols + col, (size_t)m.cols * 2u,
                         src + (size_t)src_row * src_ld + src_col, (size_t)src_ld * 2u, (size_t)cols * 2u, rows,
                         cudaMemcpyHostToDevice));
    return STARK_B200_OK;
}

stark_b200_status alloc_vector(float **dst, uint32_t padded) {
    if (*dst) return STARK_B200_OK;
    SB_TRY(dmalloc(dst, padded));
    SB_CUDA(cudaMemset(*dst, 0, (size_t)padded * 4u));
    return STARK_B200_OK;
}
stark_b200_status put_vector(float **dst, uint32_t padded, const uint16_t *src, uint32_t n) {
    SB_TRY(alloc_vector(dst, padded));
    std::vector<float> v(n);
    for (uint32_t i = 0; i < n; ++i) v[i] = bf16_bits_to_f32(src[i]);
    SB_CUDA(cudaMemcpy(*dst, v.data(), (size_t)n * 4u, cudaMemcpyHostToDevice));
    return STARK_B200_OK;
}

// Angle per position of pair i: base^(-2i / dims), or that blended with itself / factor between two pair indices (the
// "YaRN" ramp), with the factor on cos and sin that goes with it.
void rotation_table(const stark_b200_layer_desc &d, std::vector<float> &freq, float *factor) {
    const double dims = d.rot_dims;
    *factor = 1.0f;
    double lo = 0.0, hi = 0.0;
    if (d.rot_scaling == STARK_B200_ROT_YARN) {
        const double pi = 3.14159265358979323846;
        auto pair_of = [&](double turns) { return dims * log(d.rot_original / (2.0 * pi * turns)) / (2.0 * log(d.rot_base)); };
        lo = std::max(floor(pair_of(d.rot_fast)), 0.0);
        hi = std::min(ceil(pair_of(d.rot_slow)), dims - 1.0);
        *factor = (float)(0.1 * log(d.rot_factor) + 1.0);
    }
    for (uint32_t i = 0; i < d.rot_dims / 2u; ++i) {
        double f = pow(d.rot_base, -2.0 * i / dims);
        if (d.rot_scaling == STARK_B200_ROT_YARN) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f = f / d.rot_factor * ramp + f * (1.0 - ramp);
        }
        freq[i] = (float)f;
    }
}

LayerTensors &tensors_of(LayeredState *L, const Layer &layer) { return L->layers[layer.tensors].own; }

// ---- one token ------------------------------------------------------------------------------------------------------

// Spans the cached rows are divided into: about one CTA per SM, a CTA being 16 heads of a row where the tensor cores
// serve it (a power of two of spans, a few to a cluster), else one head.
void divide_cache(LatentArgs &a, uint32_t rows) {
    a.cluster = 1;
    if (!a.cache_f32 && latent_attend_mma_supports(a.s)) {
        const uint32_t ctas = (a.s.heads + 15u) / 16u * rows, most = std::max(1u, std::min(64u, 148u / ctas));
        uint32_t spans = 1;
        while (spans * 2u <= most) spans *= 2u;
        if (tunables().latent_spans) spans = std::min(spans, tunables().latent_spans);
        a.cluster = std::min(tunables().latent_cluster, spans);
        a.splits = spans / a.cluster;
    } else {
        a.splits = std::max(1u, std::min(kLatentMaxSplits, 296u / (a.s.heads * rows)));
    }
}

LatentArgs latent_args(Model *m, const Layer &layer) {
    LayeredState *L = m->layered;
    LatentArgs a{};
    a.s = layer.s;
    a.rot = layer.rot;
    a.latent_norm = tensors_of(L, layer).latent_norm;
    a.eps = L->c.eps;
    a.scale = layer.d.scale;
    a.uk_uv = tensors_of(L, layer).uk_uv;
    a.cache = layer.cache;
    a.cache_f32 = L->f32;
    a.block_table = m->block_table;
    a.num_blocks = m->num_blocks;
    a.queries = L->queries;
    a.partials = L->partials;
    a.ld_qd = tensors_of(L, layer).qd.rows;
    a.error_word = device_context()->error_word;
    return a;
}

EmbedArgs embed_args(Model *m) {
    LayeredState *L = m->layered;
    EmbedArgs e{};
    e.table = L->embed;
    e.bigram = L->bigram;
    e.buckets = L->c.bigram_buckets;
    e.width = L->c.width;
    e.vocab = L->c.vocab;
    e.mul_prev = L->c.bigram_mul_prev;
    e.mul_cur = L->c.bigram_mul_cur;
    e.scale = L->c.embed_scale;
    e.eps = L->c.eps;
    e.norm_w = L->embed_norm;
    e.history = L->history;
    return e;
}

stark_b200_status layered_issue_token(Model *m, bool full, uint32_t *launches) {
    LayeredState *L = m->layered;
    if (!device_context()) return STARK_B200_DEVICE_FAILURE;
    cudaStream_t s = m->stream;
    const bool pdl = tunables().pdl != 0u;
    uint32_t n = 0, cur = 0;
    EmbedArgs e = embed_args(m);
    e.state = m->state;
    e.x = L->x[0];
    e.m = 1;
    e.pdl = pdl;
    SB_TRY(embed_norm_launch(e, s));
    ++n;
    const float *pending = nullptr;  // norm weight of a sublayer output in y that x does not hold yet
    auto input = [&](MatvecArgs &a) {  // the residual stream, with the pending output added in the prologue
        a.x = L->x[cur];
        a.width = L->c.width;
        a.eps = L->c.eps;
        a.pdl = pdl;
        if (pending) {
            a.prologue = kRowAddNorm;
            a.y = L->y;
            a.norm_w = pending;
            a.x_out = L->x[cur ^= 1u];
            pending = nullptr;
        }
    };
    for (const Layer &layer : L->layers) {
        const LayerTensors &t = tensors_of(L, layer);
        MatvecArgs a{};
        a.w = t.qd;
        input(a);
        a.out = L->qd;
        a.out_rows = t.qd.rows;
        SB_TRY(matvec_b16_launch(a, s));
        LatentArgs la = latent_args(m, layer);
        la.qd = L->qd;
        la.state = m->state;
        la.m = 1;
        divide_cache(la, 1);
        la.out = L->attn;
        la.pdl = pdl;
        SB_TRY(latent_query_launch(la, s));
        SB_TRY(latent_attend_launch(la, s));
        SB_TRY(latent_value_launch(la, s));
        MatvecArgs o{};
        o.w = t.o;
        o.x = L->attn;
        o.out = L->y;
        o.out_rows = t.o.rows;
        o.pdl = pdl;
        SB_TRY(matvec_b16_launch(o, s));
        pending = t.norm1;
        n += 5;
        if (layer.d.feed_forward == STARK_B200_FF_NONE) continue;
        MatvecArgs g{};
        g.w = t.gate_up;
        input(g);
        g.epilogue = kRowGate;
        g.bias = t.gate_up_b;
        g.limit = layer.d.ff_limit;
        g.out = L->act;
        g.out_rows = layer.ff_p;
        SB_TRY(matvec_b16_launch(g, s));
        MatvecArgs d{};
        d.w = t.down;
        d.x = L->act;
        d.bias = t.down_b;
        d.out = L->y;
        d.out_rows = t.down.rows;
        d.pdl = pdl;
        SB_TRY(matvec_b16_launch(d, s));
        pending = t.norm2;
        n += 2;
    }
    if (full) {
        MatvecArgs h{};
        h.w = L->head;
        input(h);
        h.prologue = kRowAddNormNorm;
        h.last_w = L->final_norm;
        h.epilogue = kRowLogits;
        h.out = m->logits_f32;
        h.out_rows = L->c.vocab;
        h.partial_max = m->partial_max;
        h.partial_index = m->partial_index;
        uint32_t grid = 0;
        h.out_grid = &grid;
        SB_TRY(matvec_b16_launch(h, s));
        SB_TRY(argmax_finalize_launch(m->partial_max, m->partial_index, grid, m->state, m->generated, true, pdl, s));
        n += 2;
    } else {
        SB_TRY(ingest_advance_launch(m->state, m->pending, pdl, s));
        n += 1;
    }
    if (launches) *launches = n;
    return STARK_B200_OK;
}

// ---- a pass of rows ---------------------------------------------------------------------------------------------------

bool layered_rows_ready(Model *m) {
    LayeredState *L = m->layered;
    if (L->rows) return true;
    const uint32_t rows = std::min<uint32_t>(kPrefillBatchRows, m->num_blocks * kPageTokens);
    const size_t element = L->f32 ? 4u : 2u;
    auto bytes = [&](void **p, size_t n) { return dmalloc(reinterpret_cast<uint8_t **>(p), n) == STARK_B200_OK; };
    if (dmalloc(&m->chunk_tokens, kPrefillBatchRows + 8u) != STARK_B200_OK ||
        dmalloc(&L->rx, (size_t)rows * L->width_p) != STARK_B200_OK ||
        dmalloc(&L->ry, (size_t)rows * L->width_p) != STARK_B200_OK ||
        dmalloc(&L->rx_b16, (size_t)rows * L->width_p) != STARK_B200_OK ||
        !bytes(&L->rqd, rows * element * L->max_qd) || !bytes(&L->rattn, rows * element * L->max_attn) ||
        !bytes(&L->ract, rows * element * std::max(64u, L->max_ff)) ||
        (L->f32 && dmalloc(&L->rgu, (size_t)rows * 2u * std::max(64u, L->max_ff)) != STARK_B200_OK) ||
        dmalloc(&L->picked, kReadoutRows) != STARK_B200_OK ||
        !bytes(&L->picked_x, (size_t)kReadoutRows * L->width_p * 4u) ||
        dmalloc(&L->picked_logits, (size_t)kReadoutRows * L->c.vocab) != STARK_B200_OK)
        return false;
    L->rows = rows;
    return true;
}

// Attention of a pass over the cache, query rows in `rqd`, output rows in `rattn`.
stark_b200_status rows_attention(Model *m, const Layer &layer, uint32_t mrows, uint32_t first_pos, uint32_t *launches) {
    LayeredState *L = m->layered;
    LatentArgs a = latent_args(m, layer);
    a.qd_b16 = !L->f32;
    a.out_b16 = !L->f32;
    const size_t element = L->f32 ? 4u : 2u;
    if (!L->f32 && mrows > kPrefillSmallRows && layer.d.scale > 0.0f && latent_prefill_tc_supports(layer.s)) {
        const size_t visible = ((size_t)first_pos + mrows + kPageTokens - 1u) / kPageTokens * kPageTokens;
        if (L->expanded_rows < visible) {
            SB_CUDA(cudaStreamSynchronize(m->stream));
            cudaFree(L->expanded);
            L->expanded = nullptr;
            L->expanded_rows = 0;
            const size_t want = std::min<size_t>((size_t)m->num_blocks * kPageTokens, std::max<size_t>(visible, 4096u) * 3u / 2u);
            SB_TRY(dmalloc(&L->expanded, std::max(want, visible) * L->max_expand));
            L->expanded_rows = std::max(want, visible);
        }
        a.qd = L->rqd;
        a.first_pos = first_pos;
        a.m = mrows;
        a.splits = 1;
        a.expanded = L->expanded;
        a.out = L->rattn;
        SB_TRY(latent_rotate_append_launch(a, m->stream));
        // keys and values of every visible row; pages are handed out in order, so they are the cache's first rows
        GemmB16Args g{};
        g.w = tensors_of(L, layer).uk_uv;
        g.x = static_cast<const uint16_t *>(layer.cache);
        g.x_rows = (uint32_t)visible;
        g.m = (uint32_t)visible;
        g.ld_x = layer.s.row();
        g.kind = kGemmBf16;
        g.out = L->expanded;
        g.ld_out = g.out_cols = g.w.rows;
        SB_TRY(gemm_b16_launch(g, m->stream));
        *launches += 3;
        return latent_prefill_tc_launch(a, m->stream);
    }
    for (uint32_t r = 0; r < mrows; r += kAttendRows) {
        a.m = std::min(kAttendRows, mrows - r);
        a.first_pos = first_pos + r;
        a.qd = static_cast<const uint8_t *>(L->rqd) + (size_t)r * a.ld_qd * element;
        a.out = static_cast<uint8_t *>(L->rattn) + (size_t)r * layer.s.heads * layer.s.vdim_p * element;
        divide_cache(a, a.m);
        SB_TRY(latent_query_launch(a, m->stream));
        SB_TRY(latent_attend_launch(a, m->stream));
        SB_TRY(latent_value_launch(a, m->stream));
        *launches += 3;
    }
    return STARK_B200_OK;
}

// y = x W^T of a pass; x is the bf16 or f32 form of the rows
stark_b200_status rows_contract(Model *m, const MatrixB16 &w, const void *x, uint32_t mrows, const float *bias, void *out,
                                GemmB16Out kind, float limit, uint32_t *launches) {
    LayeredState *L = m->layered;
    ++*launches;
    if (L->f32) {
        if (kind != kGemmGate)
            return rows_gemm_f32_launch(w, static_cast<const float *>(x), mrows, bias, static_cast<float *>(out), w.rows, w.rows, m->stream);
        SB_TRY(rows_gemm_f32_launch(w, static_cast<const float *>(x), mrows, bias, L->rgu, w.rows, w.rows, m->stream));
        ++*launches;
        return clamped_gate_rows_launch(L->rgu, static_cast<float *>(out), mrows, w.rows / 2u, limit, m->stream);
    }
    GemmB16Args g{};
    g.w = w;
    g.x = static_cast<const uint16_t *>(x);
    g.x_rows = L->rows;
    g.m = mrows;
    g.ld_x = w.cols;
    g.kind = kind;
    g.out = out;
    g.out_cols = w.rows;
    g.ld_out = kind == kGemmGate ? w.rows / 2u : w.rows;
    g.bias = bias;
    g.limit = limit;
    return gemm_b16_launch(g, m->stream);
}

stark_b200_status layered_rows_pass(Model *m, const uint32_t *tokens_device, uint32_t mrows, uint32_t first_pos) {
    LayeredState *L = m->layered;
    if (!device_context()) return STARK_B200_DEVICE_FAILURE;
    if (mrows == 0 || mrows > L->rows) return STARK_B200_INVALID_ARGUMENT;
    cudaStream_t s = m->stream;
    uint32_t n = 1;
    EmbedArgs e = embed_args(m);
    e.tokens = tokens_device;
    e.first_pos = first_pos;
    e.x = L->rx;
    e.x_b16 = L->f32 ? nullptr : L->rx_b16;
    e.m = mrows;
    SB_TRY(embed_norm_launch(e, s));
    const void *x = L->f32 ? static_cast<const void *>(L->rx) : static_cast<const void *>(L->rx_b16);
    uint16_t *rounded = L->f32 ? nullptr : L->rx_b16;
    for (const Layer &layer : L->layers) {
        const LayerTensors &t = tensors_of(L, layer);
        SB_TRY(rows_contract(m, t.qd, x, mrows, nullptr, L->rqd, L->f32 ? kGemmF32 : kGemmBf16, 0.0f, &n));
        SB_TRY(rows_attention(m, layer, mrows, first_pos, &n));
        SB_TRY(rows_contract(m, t.o, L->rattn, mrows, nullptr, L->ry, kGemmF32, 0.0f, &n));
        SB_TRY(add_norm_rows_launch(L->rx, L->ry, t.norm1, mrows, L->c.width, L->c.eps, rounded, s));
        ++n;
        if (layer.d.feed_forward == STARK_B200_FF_NONE) continue;
        SB_TRY(rows_contract(m, t.gate_up, x, mrows, t.gate_up_b, L->ract, kGemmGate, layer.d.ff_limit, &n));
        SB_TRY(rows_contract(m, t.down, L->ract, mrows, t.down_b, L->ry, kGemmF32, 0.0f, &n));
        SB_TRY(add_norm_rows_launch(L->rx, L->ry, t.norm2, mrows, L->c.width, L->c.eps, rounded, s));
        ++n;
    }
    m->launches_issued += n;
    return STARK_B200_OK;
}

stark_b200_status layered_rows_logits(Model *m, const uint32_t *rows, uint32_t count, uint32_t mrows, float *dst) {
    LayeredState *L = m->layered;
    cudaStream_t s = m->stream;
    const size_t vocab = L->c.vocab;
    for (uint32_t done = 0; done < count; done += kReadoutRows) {
        const uint32_t n = std::min(kReadoutRows, count - done);
        for (uint32_t i = 0; i < n; ++i)
            if (rows[done + i] >= mrows) return STARK_B200_INVALID_ARGUMENT;
        SB_CUDA(cudaMemcpyAsync(L->picked, rows + done, n * 4u, cudaMemcpyHostToDevice, s));
        SB_TRY(norm_gather_rows_launch(L->rx, L->picked, n, L->final_norm, L->c.width, L->c.eps,
                                       L->f32 ? static_cast<float *>(L->picked_x) : nullptr,
                                       L->f32 ? nullptr : static_cast<uint16_t *>(L->picked_x), s));
        if (L->f32) {
            SB_TRY(rows_gemm_f32_launch(L->head, static_cast<const float *>(L->picked_x), n, nullptr, L->picked_logits,
                                        (uint32_t)vocab, (uint32_t)vocab, s));
        } else {
            GemmB16Args g{};
            g.w = L->head;
            g.x = static_cast<const uint16_t *>(L->picked_x);
            g.x_rows = kReadoutRows;
            g.m = n;
            g.ld_x = L->width_p;
            g.kind = kGemmF32;
            g.out = L->picked_logits;
            g.ld_out = (uint32_t)vocab;
            g.out_cols = (uint32_t)vocab;
            SB_TRY(gemm_b16_launch(g, s));
        }
        SB_CUDA(cudaMemcpyAsync(dst + done * vocab, L->picked_logits, n * vocab * 4u, cudaMemcpyDeviceToHost, s));
        SB_CUDA(cudaStreamSynchronize(s));
        m->launches_issued += 2;
    }
    return STARK_B200_OK;
}

// ---- the family -----------------------------------------------------------------------------------------------------

uint32_t layered_vocab(const Model *m) { return m->layered->c.vocab; }

stark_b200_status layered_ready(Model *m) {
    LayeredState *L = m->layered;
    uint32_t want = 1u << STARK_B200_LAYERED_EMBED | 1u << STARK_B200_LAYERED_EMBED_NORM |
                    1u << STARK_B200_LAYERED_FINAL_NORM | 1u << STARK_B200_LAYERED_HEAD;
    if (L->c.bigram_buckets) want |= 1u << STARK_B200_LAYERED_BIGRAM;
    if (L->seen != want) return STARK_B200_INVALID_STATE;
    for (uint32_t i = 0; i < L->layers.size(); ++i) {
        const Layer &layer = L->layers[i];
        if (layer.tensors != i) continue;
        uint32_t need = 0;
        for (uint32_t t = STARK_B200_LAYERED_NORM1; t <= STARK_B200_LAYERED_O; ++t) need |= 1u << t;
        if (layer.d.feed_forward != STARK_B200_FF_NONE)
            for (uint32_t t = STARK_B200_LAYERED_NORM2; t <= STARK_B200_LAYERED_DOWN_BIAS; ++t) need |= 1u << t;
        if (layer.own.seen != need) return STARK_B200_INVALID_STATE;
    }
    return STARK_B200_OK;
}

void layered_sizes(const Model *m, uint64_t *weight_bytes, uint64_t *kv_bytes_per_token) {
    const LayeredState *L = m->layered;
    uint64_t w = L->head.bytes() + (uint64_t)L->c.vocab * L->c.width * 2u +
                 (L->c.bigram_buckets ? ((uint64_t)L->c.bigram_buckets + 1u) * L->c.width * 2u : 0u), kv = 0;
    for (const Layer &l : L->layers) {
        for (const MatrixB16 *t : {&l.own.qd, &l.own.uk_uv, &l.own.o, &l.own.gate_up, &l.own.down}) w += t->bytes();
        kv += (uint64_t)l.s.row() * (L->f32 ? 4u : 2u);
    }
    *weight_bytes = w;
    *kv_bytes_per_token = kv;
}

void layered_destroy(Model *m) {
    LayeredState *L = m->layered;
    if (!L) return;
    for (Layer &l : L->layers) {
        for (MatrixB16 *t : {&l.own.qd, &l.own.uk_uv, &l.own.o, &l.own.gate_up, &l.own.down}) cudaFree(t->data);
        for (float *p : {l.own.latent_norm, l.own.norm1, l.own.norm2, l.own.gate_up_b, l.own.down_b, l.freq}) cudaFree(p);
        cudaFree(l.cache);
    }
    for (void *p : {(void *)L->embed, (void *)L->bigram, (void *)L->head.data, (void *)L->embed_norm, (void *)L->final_norm,
                    (void *)L->history, (void *)L->x[0], (void *)L->x[1], (void *)L->y, (void *)L->qd, (void *)L->attn,
                    (void *)L->act, (void *)L->queries, (void *)L->partials, (void *)L->rx, (void *)L->ry, (void *)L->rx_b16,
                    L->rqd, L->rattn, L->ract, (void *)L->rgu, (void *)L->expanded, (void *)L->picked, L->picked_x,
                    (void *)L->picked_logits})
        cudaFree(p);
    delete L;
    m->layered = nullptr;
}

ModelFamily make_layered_family() {
    ModelFamily f{};
    f.name = "layered";
    f.min_rows = 1;
    f.input_vocab = layered_vocab;
    f.ready = layered_ready;
    f.issue_token = layered_issue_token;
    f.rows_ready = layered_rows_ready;
    f.rows_pass = layered_rows_pass;
    f.rows_logits = layered_rows_logits;
    f.sizes = layered_sizes;
    f.destroy = layered_destroy;
    return f;
}
const ModelFamily kLayeredFamily = make_layered_family();

stark_b200_status check_layer(const stark_b200_layer_desc &d) {
    if (d.struct_size != sizeof(d)) return STARK_B200_ABI_MISMATCH;
    if (d.mixer != STARK_B200_MIXER_LATENT || d.feed_forward > STARK_B200_FF_CLAMPED_GATE || d.rot_scaling > STARK_B200_ROT_YARN)
        return STARK_B200_UNSUPPORTED;
    if (!d.heads || !d.dim || !d.vdim || !d.kv_rank || d.rot_dim % 2u || d.rot_dims % 2u || d.rot_dims > d.rot_dim ||
        !std::isfinite(d.scale) || !(d.rot_base > 0.0) ||
        (d.rot_scaling == STARK_B200_ROT_YARN && !(d.rot_factor > 0.0 && d.rot_original > 0.0 && d.rot_fast > 0.0 && d.rot_slow > 0.0)) ||
        (d.feed_forward == STARK_B200_FF_CLAMPED_GATE && !d.ff_width))
        return STARK_B200_INVALID_ARGUMENT;
    return STARK_B200_OK;
}

stark_b200_status build_layers(Model *m, const stark_b200_layer_desc *descs) {
    LayeredState *L = m->layered;
    L->layers.resize(L->c.layers);
    for (uint32_t i = 0; i < L->c.layers; ++i) {
        Layer &l = L->layers[i];
        l.d = descs[i];
        SB_TRY(check_layer(l.d));
        l.tensors = i;
        if (l.d.weights_of != UINT32_MAX) {
            if (l.d.weights_of >= L->c.layers || descs[l.d.weights_of].weights_of != UINT32_MAX) return STARK_B200_INVALID_ARGUMENT;
            // everything but the reference must equal the layer it points to
            stark_b200_layer_desc a = l.d, b = descs[l.d.weights_of];
            a.weights_of = b.weights_of = 0;
            if (memcmp(&a, &b, sizeof a) != 0) return STARK_B200_INVALID_ARGUMENT;
            l.tensors = l.d.weights_of;
        }
        LatentShape &s = l.s;
        s.heads = l.d.heads, s.dim = l.d.dim, s.rot_dim = l.d.rot_dim, s.vdim = l.d.vdim, s.rank = l.d.kv_rank;
        s.dim_p = pad64(s.dim), s.rot_p = pad64(s.rot_dim), s.vdim_p = pad64(s.vdim), s.rank_p = pad64(s.rank);
        if (!latent_shape_supported(s)) return STARK_B200_UNSUPPORTED;
        l.ff_p = l.d.feed_forward == STARK_B200_FF_NONE ? 0u : pad64(l.d.ff_width);
        std::vector<float> freq(std::max(1u, s.rot_p / 2u), 0.0f);
        rotation_table(l.d, freq, &l.rot.factor);
        SB_TRY(dmalloc(&l.freq, freq.size()));
        SB_CUDA(cudaMemcpy(l.freq, freq.data(), freq.size() * 4u, cudaMemcpyHostToDevice));
        l.rot.freq = l.freq;
        l.rot.pairs = l.d.rot_dims / 2u;
        const size_t cache = (size_t)m->num_blocks * kPageTokens * s.row() * (L->f32 ? 4u : 2u);
        SB_CUDA(cudaMalloc(&l.cache, cache));
        SB_CUDA(cudaMemset(l.cache, 0, cache));
        L->max_qd = std::max(L->max_qd, s.q_width() + s.row());
        L->max_attn = std::max(L->max_attn, s.heads * s.vdim_p);
        L->max_ff = std::max(L->max_ff, l.ff_p);
        L->max_expand = std::max(L->max_expand, s.heads * (s.dim_p + s.vdim_p));
        L->query_floats = std::max(L->query_floats, (size_t)kAttendRows * s.heads * s.row());
        for (uint32_t r = 1; r <= kAttendRows; ++r) {
            LatentArgs probe{};
            probe.s = s;
            probe.cache_f32 = L->f32;
            divide_cache(probe, r);
            L->partial_floats = std::max(L->partial_floats, latent_partial_floats(s, r, probe.splits * probe.cluster));
        }
    }
    for (const MatrixB16 probe : {MatrixB16{nullptr, 1, L->width_p}, MatrixB16{nullptr, 1, L->max_attn},
                                  MatrixB16{nullptr, 1, std::max(64u, L->max_ff)}})
        if (!matvec_b16_supports(probe)) return STARK_B200_UNSUPPORTED;
    SB_TRY(dmalloc(&L->history, (size_t)m->num_blocks * kPageTokens + 1u));
    for (float **p : {&L->x[0], &L->x[1], &L->y}) SB_TRY(dmalloc(p, L->width_p));
    SB_TRY(dmalloc(&L->qd, L->max_qd));
    SB_TRY(dmalloc(&L->attn, L->max_attn));
    SB_TRY(dmalloc(&L->act, std::max(64u, L->max_ff)));
    SB_TRY(dmalloc(&L->queries, L->query_floats));
    return dmalloc(&L->partials, L->partial_floats);
}

stark_b200_status layered_create(const stark_b200_layered_config &c, const stark_b200_layer_desc *descs, Model **out) {
    *out = nullptr;
    if (!c.vocab || !c.width || !c.layers || !c.context_tokens || c.width > 32768u || !(c.eps >= 0.0f) ||
        c.compute > STARK_B200_F32 || (uint64_t)c.bigram_buckets + 1u > UINT32_MAX || c.bigram_mul_prev > UINT32_MAX ||
        c.bigram_mul_cur > UINT32_MAX)
        return STARK_B200_INVALID_ARGUMENT;
    if (!device_context()) return STARK_B200_DEVICE_FAILURE;
    Model *m = new (std::nothrow) Model();
    LayeredState *L = new (std::nothrow) LayeredState();
    if (!m || !L) {
        delete m;
        delete L;
        return STARK_B200_OUT_OF_MEMORY;
    }
    m->family = &kLayeredFamily;
    m->layered = L;
    L->c = c;
    L->width_p = pad64(c.width);
    L->f32 = c.compute == STARK_B200_F32;
    m->cfg.layers = c.layers;
    m->cfg.hidden = c.width;
    m->cfg.vocab = c.vocab;
    m->cfg.context_tokens = c.context_tokens;
    m->cfg.eps = c.eps;
    stark_b200_status st = model_create_session(m, true);
    if (st == STARK_B200_OK) st = build_layers(m, descs);
    if (st != STARK_B200_OK) {
        delete m;
        return st;
    }
    *out = m;
    return STARK_B200_OK;
}

stark_b200_status layered_set(Model *m, uint32_t layer, uint32_t which, const uint16_t *src, uint32_t rows, uint32_t cols) {
    LayeredState *L = m->layered;
    if (m->finalized) return STARK_B200_INVALID_STATE;
    const auto &c = L->c;
    auto shaped = [&](uint32_t r, uint32_t k) { return rows == r && cols == k; };
    if (which <= STARK_B200_LAYERED_HEAD) {
        switch (which) {
            case STARK_B200_LAYERED_EMBED:
            case STARK_B200_LAYERED_BIGRAM: {
                const bool bigram = which == STARK_B200_LAYERED_BIGRAM;
                if (!shaped(bigram ? c.bigram_buckets + 1u : c.vocab, c.width) || (bigram && !c.bigram_buckets))
                    return STARK_B200_INVALID_ARGUMENT;
                uint16_t **dst = bigram ? &L->bigram : &L->embed;
                if (!*dst) SB_TRY(dmalloc(dst, (size_t)rows * cols));
                SB_CUDA(cudaMemcpy(*dst, src, (size_t)rows * cols * 2u, cudaMemcpyHostToDevice));
                break;
            }
            case STARK_B200_LAYERED_EMBED_NORM:
            case STARK_B200_LAYERED_FINAL_NORM:
                if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
                SB_TRY(put_vector(which == STARK_B200_LAYERED_EMBED_NORM ? &L->embed_norm : &L->final_norm, L->width_p, src, cols));
                break;
            default:
                if (!shaped(c.vocab, c.width)) return STARK_B200_INVALID_ARGUMENT;
                SB_TRY(alloc_matrix(L->head, c.vocab, L->width_p));
                SB_TRY(place(L->head, 0, 0, src, cols, 0, 0, rows, cols));
        }
        L->seen |= 1u << which;
        return STARK_B200_OK;
    }
    if (layer >= L->layers.size() || which > STARK_B200_LAYERED_DOWN_BIAS) return STARK_B200_INVALID_ARGUMENT;
    Layer &l = L->layers[layer];
    if (l.tensors != layer) return STARK_B200_INVALID_ARGUMENT;  // this layer has no tensors of its own
    if (which >= STARK_B200_LAYERED_NORM2 && l.d.feed_forward == STARK_B200_FF_NONE) return STARK_B200_INVALID_ARGUMENT;
    const LatentShape &s = l.s;
    LayerTensors &t = l.own;
    switch (which) {
        case STARK_B200_LAYERED_NORM1:
        case STARK_B200_LAYERED_NORM2:
            if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(which == STARK_B200_LAYERED_NORM1 ? &t.norm1 : &t.norm2, L->width_p, src, cols));
            break;
        case STARK_B200_LAYERED_Q:
            if (!shaped(s.heads * (s.dim + s.rot_dim), c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.qd, s.q_width() + s.row(), L->width_p));
            for (uint32_t h = 0; h < s.heads; ++h) {
                SB_TRY(place(t.qd, h * s.q_head(), 0, src, cols, h * (s.dim + s.rot_dim), 0, s.dim, cols));
                if (s.rot_dim)
                    SB_TRY(place(t.qd, h * s.q_head() + s.dim_p, 0, src, cols, h * (s.dim + s.rot_dim) + s.dim, 0, s.rot_dim, cols));
            }
            break;
        case STARK_B200_LAYERED_DKV:
            if (!shaped(s.rank + s.rot_dim, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.qd, s.q_width() + s.row(), L->width_p));
            SB_TRY(place(t.qd, s.q_width(), 0, src, cols, 0, 0, s.rank, cols));
            if (s.rot_dim) SB_TRY(place(t.qd, s.q_width() + s.rank_p, 0, src, cols, s.rank, 0, s.rot_dim, cols));
            break;
        case STARK_B200_LAYERED_DKV_NORM:
            if (!shaped(1, s.rank)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(&t.latent_norm, s.rank_p, src, cols));
            break;
        case STARK_B200_LAYERED_UK:
        case STARK_B200_LAYERED_UV: {
            const bool key = which == STARK_B200_LAYERED_UK;
            const uint32_t n = key ? s.dim : s.vdim, n_p = key ? s.dim_p : s.vdim_p;
            if (!shaped(s.heads * n, s.rank)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.uk_uv, s.heads * (s.dim_p + s.vdim_p), s.rank_p));
            for (uint32_t h = 0; h < s.heads; ++h)
                SB_TRY(place(t.uk_uv, (key ? 0u : s.heads * s.dim_p) + h * n_p, 0, src, cols, h * n, 0, n, cols));
            break;
        }
        case STARK_B200_LAYERED_O:
            if (!shaped(c.width, s.heads * s.vdim)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.o, L->width_p, s.heads * s.vdim_p));
            for (uint32_t h = 0; h < s.heads; ++h) SB_TRY(place(t.o, 0, h * s.vdim_p, src, cols, 0, h * s.vdim, rows, s.vdim));
            break;
        case STARK_B200_LAYERED_GATE:
        case STARK_B200_LAYERED_UP:
            if (!shaped(l.d.ff_width, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.gate_up, 2u * l.ff_p, L->width_p));
            for (uint32_t r = 0; r < rows; r += 16u)
                SB_TRY(place(t.gate_up, pair_row(r, which == STARK_B200_LAYERED_UP), 0, src, cols, r, 0, std::min(16u, rows - r), cols));
            break;
        case STARK_B200_LAYERED_GATE_BIAS:
        case STARK_B200_LAYERED_UP_BIAS: {
            if (!shaped(1, l.d.ff_width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_vector(&t.gate_up_b, 2u * l.ff_p));
            std::vector<float> v(2u * l.ff_p);
            SB_CUDA(cudaMemcpy(v.data(), t.gate_up_b, v.size() * 4u, cudaMemcpyDeviceToHost));  // the other half may be there
            for (uint32_t r = 0; r < cols; ++r) v[pair_row(r, which == STARK_B200_LAYERED_UP_BIAS)] = bf16_bits_to_f32(src[r]);
            SB_CUDA(cudaMemcpy(t.gate_up_b, v.data(), v.size() * 4u, cudaMemcpyHostToDevice));
            break;
        }
        case STARK_B200_LAYERED_DOWN:
            if (!shaped(c.width, l.d.ff_width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(alloc_matrix(t.down, L->width_p, l.ff_p));
            SB_TRY(place(t.down, 0, 0, src, cols, 0, 0, rows, cols));
            break;
        case STARK_B200_LAYERED_DOWN_BIAS:
            if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(&t.down_b, L->width_p, src, cols));
            break;
        default: return STARK_B200_INVALID_ARGUMENT;
    }
    t.seen |= 1u << which;
    return STARK_B200_OK;
}

}  // namespace

}  // namespace sb

using namespace sb;

extern "C" {

stark_b200_status stark_b200_layered_create(const stark_b200_layered_config *config, const stark_b200_layer_desc *layers,
                                            stark_b200_model **out_model) {
    if (!config || !layers || !out_model) return STARK_B200_INVALID_ARGUMENT;
    *out_model = nullptr;
    if (config->struct_size != sizeof(*config) || config->abi_version != STARK_B200_ABI_VERSION) return STARK_B200_ABI_MISMATCH;
    Model *m = nullptr;
    SB_TRY(layered_create(*config, layers, &m));
    *out_model = reinterpret_cast<stark_b200_model *>(m);
    return STARK_B200_OK;
}

stark_b200_status stark_b200_layered_set_tensor(stark_b200_model *model, uint32_t layer, uint32_t which, const void *data_bf16,
                                                uint32_t rows, uint32_t columns) {
    Model *m = reinterpret_cast<Model *>(model);
    if (!m || !m->layered || !data_bf16) return STARK_B200_INVALID_ARGUMENT;
    return layered_set(m, layer, which, static_cast<const uint16_t *>(data_bf16), rows, columns);
}

}  // extern "C"
