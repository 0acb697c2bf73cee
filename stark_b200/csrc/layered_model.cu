// The layered family: decoders whose configuration lists every layer's mixer and feed-forward.  Two mixers (latent
// attention; grouped-query attention with short convolutions), two gated feed-forwards, two arrangements of a layer, an
// embedding with or without a hashed bigram table and a norm, a read-out of its own or tied to the embedding, layers that
// use another layer's tensors: Guvulorn and Pomelix are choices among them.  This file holds what such a model owns --
// tensors in the padded layout of layered.cuh, a cache per layer over the session's page table, the state of the
// convolutions, the token history -- and what one token and one pass of prompt rows launch; stepping, recording, prompt
// loop, read-out, sampling and rewind are the shared token loop's.
//
// Arrangement "post-norm": x += norm1(mixer(x)), x += norm2(ff(x)).  A token's layer:
//   u = W x                               matvec; the residual add of the sublayer before it in the prologue
//   mixer                                 latent: query, attend, value; grouped: one launch
//   y = W_o attn                          matvec
//   act = gate(W_gu x)                    matvec, x = x + norm1(y) in the prologue, biases and gate in the epilogue
//   y = W_down act                        matvec
// and the read-out matvec forms x + norm2(y) and the last norm in its prologue and the greedy pick in its epilogue.
// Arrangement "parallel": h = norm1(x), x += mult * (scale1 * mixer(h) + scale2 * ff(h)).  A token's layer:
//   [u | act] = [W; gate of W_gu] h       one matvec, the norm in its prologue, the gate in its epilogue
//   mixer
//   x += scale1 * W_o attn + scale2 * W_down act      one matvec over both inputs, the residual add in its epilogue
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
    // in: the mixer's projections of the layer's input (parallel: gate and up rows behind them); parallel: out = o and
    // down side by side.  gate_up, o and down are runs of those then, matrices of their own otherwise.
    MatrixB16 in, out, uk_uv, gate_up, o, down;
    float *latent_norm = nullptr, *norm1 = nullptr, *norm2 = nullptr, *gate_up_b = nullptr, *down_b = nullptr;
    float *conv_w = nullptr;                            // [taps][width of the projected row]
    float *scale1 = nullptr, *scale2 = nullptr;         // times residual_mult
    float share = 0.0f;
    uint32_t seen = 0;  // bit per tensor id
};
struct Layer {
    stark_b200_layer_desc d{};
    LatentShape s{};    // STARK_B200_MIXER_LATENT
    Rotation rot{};
    float *freq = nullptr;
    void *cache = nullptr;
    GroupedShape g{};   // STARK_B200_MIXER_GROUPED
    uint32_t taps = 0;  // at least 1: a layer without convolutions has the factor 1 on every channel
    void *keys = nullptr, *values = nullptr, *recent = nullptr, *tails = nullptr;
    ValueMix mix = kMixNone;
    uint32_t ff_p = 0;
    uint32_t tensors = 0;  // index of the layer that holds them
    LayerTensors own;
    bool latent() const { return d.mixer == STARK_B200_MIXER_LATENT; }
    uint32_t mixer_width() const { return latent() ? s.q_width() + s.row() : g.width(); }          // projected row
    uint32_t attn_width() const { return latent() ? s.heads * s.vdim_p : g.heads * g.vdim_p; }     // attention output row
    Gate gate() const { return {d.feed_forward == STARK_B200_FF_SILU_GATE ? kGateSilu : kGateClamped, d.ff_limit}; }
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
    bool parallel = false;
    // widest rows over the layers
    uint32_t max_in = 0, max_mixer = 0, max_attn = 0, max_ff = 0, max_joint = 0, max_expand = 0, max_q = 0, max_first = 0;
    size_t query_floats = 0, partial_floats = 0;
    // one token; attn: attention output with the gated activation behind it
    float *x[2] = {nullptr, nullptr}, *y = nullptr, *u = nullptr, *attn = nullptr;
    float *queries = nullptr, *partials = nullptr, *first_values = nullptr;
    // a pass of rows
    uint32_t rows = 0;
    float *rx = nullptr, *ry = nullptr;
    void *rh = nullptr;                                      // what the contractions read: x or its norm, bf16 or f32
    void *ru = nullptr, *rattn = nullptr, *ract = nullptr;   // bf16, or f32 in the 32-bit form
    uint16_t *rq = nullptr;                                  // finished queries of the grouped mixer, bf16 form only
    float *rfirst = nullptr;
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
    SB_CUDA(cudaMemcpy2D(m.data + (size_t)row * m.pitch() + col, (size_t)m.pitch() * 2u,
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
stark_b200_status put_vector(float **dst, uint32_t padded, const uint16_t *src, uint32_t n, float offset = 0.0f, float factor = 1.0f) {
    SB_TRY(alloc_vector(dst, padded));
    std::vector<float> v(n);
    for (uint32_t i = 0; i < n; ++i) v[i] = (offset + bf16_bits_to_f32(src[i])) * factor;
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
        a.splits = std::max(1u, std::min(kMaxSplits, 296u / (a.s.heads * rows)));
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
    a.ld_qd = layer.mixer_width();
    a.error_word = device_context()->error_word;
    return a;
}

// Spans of the grouped decode attention: a cluster of up to eight CTAs (8 query heads of a key / value head each), which
// merges them; several clusters, merged by a launch of their own, where heads are few and the context is long.
void divide_grouped(const Model *m, GroupedArgs &a) {
    const uint32_t tiles = a.s.groups * ((a.s.per() + kGroupedHeadTile - 1u) / kGroupedHeadTile), pages = m->num_blocks;
    // the contraction before it: two CTAs an SM, an input row and some words each
    a.beside_smem = 2u * ((m->layered->width_p + 255u) / 256u * 1024u + 2048u);
    a.cluster = 1;
    while (a.cluster < 8u && a.cluster * 2u * tiles <= 148u && a.cluster < pages) a.cluster *= 2u;
    if (tunables().grouped_cluster) a.cluster = tunables().grouped_cluster;
    a.splits = std::max(1u, std::min({148u / (a.cluster * tiles), pages / (a.cluster * 16u), kMaxSplits}));
    if (tunables().grouped_splits) a.splits = tunables().grouped_splits;
}

GroupedArgs grouped_args(Model *m, const Layer &layer) {
    LayeredState *L = m->layered;
    const LayerTensors &t = tensors_of(L, layer);
    GroupedArgs a{};
    a.s = layer.g;
    a.conv = {t.conv_w, layer.taps, layer.recent, layer.tails};
    a.ld_u = layer.mixer_width();
    a.eps = L->c.eps, a.scale = layer.d.scale;
    a.temp_coef = layer.d.q_temp_coef, a.temp_every = layer.d.q_temp_every;
    a.mix = layer.mix, a.share = t.share;
    a.keys = layer.keys, a.values = layer.values;
    a.cache_f32 = L->f32;
    a.block_table = m->block_table, a.num_blocks = m->num_blocks;
    a.partials = L->partials;
    a.splits = a.cluster = 1;
    a.error_word = device_context()->error_word;
    return a;
}

// The span attention over this layer's cache, behind grouped_rows.
SpanAttendArgs span_args(const GroupedArgs &g, void *out, bool out_b16) {
    SpanAttendArgs a{};
    a.queries = g.queries;
    a.heads = g.s.heads, a.key_heads = g.s.groups, a.width = g.s.dim_p, a.out_width = g.s.vdim_p;
    a.keys = g.keys, a.values = g.values, a.key_pitch = g.s.dim_p, a.value_pitch = g.s.vdim_p;
    a.cache_f32 = g.cache_f32;
    a.block_table = g.block_table, a.state = g.state, a.first_pos = g.first_pos, a.m = g.m;
    a.splits = g.splits;
    a.partials = g.partials;
    a.out = out, a.ld_out = g.s.heads * g.s.vdim_p, a.out_b16 = out_b16;
    a.pdl = g.pdl;
    return a;
}
uint32_t plain_splits(const GroupedShape &s, uint32_t rows) { return std::max(1u, std::min(kMaxSplits, 296u / (s.heads * rows))); }

EmbedArgs embed_args(Model *m) {
    LayeredState *L = m->layered;
    EmbedArgs e{};
    const bool tied = (L->c.flags & STARK_B200_LAYERED_TIED_HEAD) != 0u;
    e.table = tied ? L->head.data : L->embed;
    e.ld_table = tied ? L->width_p : L->c.width;
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

// A layer's mixer for one token: projected row in `u`, attention output to `attn`.
stark_b200_status token_mixer(Model *m, const Layer &layer, uint32_t *launches) {
    LayeredState *L = m->layered;
    cudaStream_t s = m->stream;
    const bool pdl = tunables().pdl != 0u;
    if (layer.latent()) {
        LatentArgs a = latent_args(m, layer);
        a.qd = L->u;
        a.state = m->state;
        a.m = 1;
        divide_cache(a, 1);
        a.out = L->attn;
        a.pdl = pdl;
        SB_TRY(latent_query_launch(a, s));
        SB_TRY(latent_attend_launch(a, s));
        *launches += 3;
        return latent_value_launch(a, s);
    }
    GroupedArgs a = grouped_args(m, layer);
    a.u = L->u;
    a.first_values = L->first_values;
    a.state = m->state;
    a.m = 1;
    a.pdl = pdl;
    if (!L->f32 && grouped_attend_mma_supports(layer.g)) {
        divide_grouped(m, a);
        a.out = L->attn;
        SB_TRY(grouped_attend_mma_launch(a, s));
        ++*launches;
        if (a.splits == 1u) return STARK_B200_OK;
    } else {
        a.queries = L->queries;
        a.splits = plain_splits(layer.g, 1);
        SB_TRY(grouped_rows_launch(a, s));
        SB_TRY(span_attend_launch(span_args(a, nullptr, false), s));
        *launches += 2;
    }
    ++*launches;
    return span_merge_launch(span_args(a, L->attn, false), s);
}

stark_b200_status token_parallel_layer(Model *m, const Layer &layer, uint32_t *launches) {
    LayeredState *L = m->layered;
    const LayerTensors &t = tensors_of(L, layer);
    const bool pdl = tunables().pdl != 0u, ff = layer.d.feed_forward != STARK_B200_FF_NONE;
    MatvecArgs a{};
    a.w = t.in;
    a.prologue = kRowNorm;
    a.x = L->x[0];
    a.norm_w = t.norm1;
    a.width = L->c.width;
    a.eps = L->c.eps;
    a.pdl = pdl;
    if (ff) {
        a.epilogue = kRowGate;
        a.gate = layer.gate();
        a.stored_rows = layer.mixer_width();
        a.stored_out = L->u;
        a.out = L->attn + layer.attn_width();
    } else {
        a.out = L->u;
        a.out_rows = t.in.rows;
    }
    SB_TRY(matvec_b16_launch(a, m->stream));
    SB_TRY(token_mixer(m, layer, launches));
    MatvecArgs o{};
    o.w = t.out;
    o.epilogue = kRowResidual;
    o.x = L->attn;
    o.residual = o.out = L->x[0];
    o.scale_a = t.scale1;
    o.scale_b = t.scale2;
    o.split_col = layer.attn_width();
    o.out_rows = t.out.rows;
    o.pdl = pdl;
    *launches += 2;
    return matvec_b16_launch(o, m->stream);
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
        if (L->parallel) {
            SB_TRY(token_parallel_layer(m, layer, &n));
            continue;
        }
        const LayerTensors &t = tensors_of(L, layer);
        MatvecArgs a{};
        a.w = t.in;
        input(a);
        a.out = L->u;
        a.out_rows = t.in.rows;
        SB_TRY(matvec_b16_launch(a, s));
        SB_TRY(token_mixer(m, layer, &n));
        MatvecArgs o{};
        o.w = t.o;
        o.x = L->attn;
        o.out = L->y;
        o.out_rows = t.o.rows;
        o.pdl = pdl;
        SB_TRY(matvec_b16_launch(o, s));
        pending = t.norm1;
        n += 2;
        if (layer.d.feed_forward == STARK_B200_FF_NONE) continue;
        float *act = L->attn + layer.attn_width();
        MatvecArgs g{};
        g.w = t.gate_up;
        input(g);
        g.epilogue = kRowGate;
        g.bias = t.gate_up_b;
        g.gate = layer.gate();
        g.out = act;
        SB_TRY(matvec_b16_launch(g, s));
        MatvecArgs d{};
        d.w = t.down;
        d.x = act;
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
        h.prologue = L->parallel ? kRowNorm : kRowAddNormNorm;
        if (L->parallel) h.norm_w = L->final_norm;
        else h.last_w = L->final_norm;
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
    // the 32-bit form leaves a fused contraction's gate and up columns beside the projected row; the bf16 form never does
    if (dmalloc(&m->chunk_tokens, kPrefillBatchRows + 8u) != STARK_B200_OK ||
        dmalloc(&L->rx, (size_t)rows * L->width_p) != STARK_B200_OK ||
        (!L->parallel && dmalloc(&L->ry, (size_t)rows * L->width_p) != STARK_B200_OK) ||
        ((L->parallel || !L->f32) && !bytes(&L->rh, rows * element * L->width_p)) ||
        !bytes(&L->ru, rows * element * (L->f32 ? L->max_in : L->max_mixer)) || !bytes(&L->rattn, rows * element * L->max_attn) ||
        !bytes(&L->ract, rows * element * std::max(64u, L->max_ff)) ||
        (!L->f32 && L->max_q && dmalloc(&L->rq, (size_t)rows * L->max_q) != STARK_B200_OK) ||
        (L->max_first && dmalloc(&L->rfirst, (size_t)rows * L->max_first) != STARK_B200_OK) ||
        (L->f32 && !L->parallel && dmalloc(&L->rgu, (size_t)rows * 2u * std::max(64u, L->max_ff)) != STARK_B200_OK) ||
        dmalloc(&L->picked, kReadoutRows) != STARK_B200_OK ||
        !bytes(&L->picked_x, (size_t)kReadoutRows * L->width_p * 4u) ||
        dmalloc(&L->picked_logits, (size_t)kReadoutRows * L->c.vocab) != STARK_B200_OK)
        return false;
    L->rows = rows;
    return true;
}

// Attention of a pass over the cache, projected rows in `ru` (ld_u apart), output rows in `rattn`.
stark_b200_status rows_latent(Model *m, const Layer &layer, uint32_t ld_u, uint32_t mrows, uint32_t first_pos, uint32_t *launches) {
    LayeredState *L = m->layered;
    LatentArgs a = latent_args(m, layer);
    a.ld_qd = ld_u;
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
        a.qd = L->ru;
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
        a.qd = static_cast<const uint8_t *>(L->ru) + (size_t)r * a.ld_qd * element;
        a.out = static_cast<uint8_t *>(L->rattn) + (size_t)r * layer.attn_width() * element;
        divide_cache(a, a.m);
        SB_TRY(latent_query_launch(a, m->stream));
        SB_TRY(latent_attend_launch(a, m->stream));
        SB_TRY(latent_value_launch(a, m->stream));
        *launches += 3;
    }
    return STARK_B200_OK;
}

stark_b200_status rows_grouped(Model *m, const Layer &layer, uint32_t ld_u, uint32_t mrows, uint32_t first_pos, uint32_t *launches) {
    LayeredState *L = m->layered;
    const GroupedShape &s = layer.g;
    GroupedArgs a = grouped_args(m, layer);
    a.u_b16 = !L->f32;
    a.ld_u = ld_u;
    if (!L->f32 && layer.d.scale > 0.0f && attend_tc_supports(s.dim_p / 64u, s.vdim_p / 64u)) {
        a.u = L->ru;
        a.first_values = L->rfirst;
        a.first_pos = first_pos;
        a.m = mrows;
        a.queries_b16 = L->rq;
        SB_TRY(grouped_rows_launch(a, m->stream));
        AttendTcArgs t{};
        const uint32_t cached = m->num_blocks * s.groups * kPageTokens;
        t.queries = L->rq;
        t.ld_q = s.heads * s.dim_p, t.heads = s.heads, t.key_heads = s.groups;
        t.keys = {static_cast<const uint16_t *>(layer.keys), s.dim_p, cached, s.dim_p, 0u, 0u};
        t.values = {static_cast<const uint16_t *>(layer.values), s.vdim_p, cached, s.vdim_p, 0u, 0u};
        t.own_blocks = s.dim_p / 64u, t.value_blocks = s.vdim_p / 64u;
        t.block_table = m->block_table;
        t.first_pos = first_pos, t.m = mrows;
        t.scale = layer.d.scale;
        t.dim_bound = (float)s.dim;  // a query (without its temperature) and a key have norms of sqrt(dim) at most
        t.temp_coef = a.temp_coef, t.temp_every = a.temp_every;
        t.out = static_cast<uint16_t *>(L->rattn);
        t.error_word = a.error_word;
        *launches += mrows > kConvSpare && layer.taps > 1u ? 3u : 2u;
        return attend_tc_launch(t, m->stream);
    }
    const size_t element = L->f32 ? 4u : 2u;
    a.queries = L->queries;
    for (uint32_t r = 0; r < mrows; r += kAttendRows) {
        a.m = std::min(kAttendRows, mrows - r);
        a.first_pos = first_pos + r;
        a.u = static_cast<const uint8_t *>(L->ru) + (size_t)r * ld_u * element;
        a.first_values = L->rfirst ? L->rfirst + (size_t)r * s.groups * s.vdim : nullptr;
        a.splits = plain_splits(s, a.m);
        const SpanAttendArgs span =
            span_args(a, static_cast<uint8_t *>(L->rattn) + (size_t)r * layer.attn_width() * element, !L->f32);
        SB_TRY(grouped_rows_launch(a, m->stream));
        SB_TRY(span_attend_launch(span, m->stream));
        SB_TRY(span_merge_launch(span, m->stream));
        *launches += a.m > kConvSpare && layer.taps > 1u ? 4u : 3u;
    }
    return STARK_B200_OK;
}

stark_b200_status rows_mixer(Model *m, const Layer &layer, uint32_t ld_u, uint32_t mrows, uint32_t first_pos, uint32_t *launches) {
    return layer.latent() ? rows_latent(m, layer, ld_u, mrows, first_pos, launches)
                          : rows_grouped(m, layer, ld_u, mrows, first_pos, launches);
}

// y = x W^T of a pass; x is the bf16 or f32 form of the rows
stark_b200_status rows_contract(Model *m, const MatrixB16 &w, const void *x, uint32_t mrows, const float *bias, void *out,
                                GemmB16Out kind, Gate gate, uint32_t *launches) {
    LayeredState *L = m->layered;
    ++*launches;
    if (L->f32) {
        if (kind != kGemmGate)
            return rows_gemm_f32_launch(w, static_cast<const float *>(x), mrows, bias, static_cast<float *>(out), w.rows, w.rows, m->stream);
        SB_TRY(rows_gemm_f32_launch(w, static_cast<const float *>(x), mrows, bias, L->rgu, w.rows, w.rows, m->stream));
        ++*launches;
        return gate_rows_launch(L->rgu, w.rows, static_cast<float *>(out), mrows, w.rows / 2u, gate, m->stream);
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
    g.gate = gate;
    return gemm_b16_launch(g, m->stream);
}

// x += scale * (in W^T) of a pass
stark_b200_status rows_add_contract(Model *m, const MatrixB16 &w, const void *in, uint32_t mrows, const float *scale, uint32_t *launches) {
    LayeredState *L = m->layered;
    ++*launches;
    if (L->f32)
        return rows_gemm_f32_launch(w, static_cast<const float *>(in), mrows, nullptr, L->rx, L->width_p, w.rows, m->stream, scale);
    GemmB16Args g{};
    g.w = w;
    g.x = static_cast<const uint16_t *>(in);
    g.x_rows = L->rows;
    g.m = mrows;
    g.ld_x = w.cols;
    g.kind = kGemmResidual;
    g.out = L->rx;
    g.ld_out = L->width_p;
    g.out_cols = w.rows;
    g.scale = scale;
    return gemm_b16_launch(g, m->stream);
}

stark_b200_status rows_parallel_layer(Model *m, const Layer &layer, uint32_t mrows, uint32_t first_pos, uint32_t *launches) {
    LayeredState *L = m->layered;
    const LayerTensors &t = tensors_of(L, layer);
    const bool ff = layer.d.feed_forward != STARK_B200_FF_NONE;
    const uint32_t mixer = layer.mixer_width();
    uint32_t ld_u = mixer;
    SB_TRY(norm_rows_launch(L->rx, nullptr, mrows, t.norm1, L->c.width, L->c.eps, L->f32 ? static_cast<float *>(L->rh) : nullptr,
                            L->f32 ? nullptr : static_cast<uint16_t *>(L->rh), m->stream));
    if (L->f32) {
        float *u = static_cast<float *>(L->ru);
        ld_u = t.in.rows;
        SB_TRY(rows_gemm_f32_launch(t.in, static_cast<const float *>(L->rh), mrows, nullptr, u, ld_u, ld_u, m->stream));
        if (ff) SB_TRY(gate_rows_launch(u + mixer, ld_u, static_cast<float *>(L->ract), mrows, layer.ff_p, layer.gate(), m->stream));
        *launches += ff ? 3u : 2u;
    } else {
        GemmB16Args g{};
        g.w = t.in;
        g.x = static_cast<const uint16_t *>(L->rh);
        g.x_rows = L->rows;
        g.m = mrows;
        g.ld_x = t.in.cols;
        g.out_cols = t.in.rows;
        if (ff) {
            g.kind = kGemmGate;
            g.gate = layer.gate();
            g.stored_cols = g.ld_stored = mixer;
            g.stored_out = static_cast<uint16_t *>(L->ru);
            g.out = L->ract;
            g.ld_out = layer.ff_p;
        } else {
            g.kind = kGemmBf16;
            g.out = L->ru;
            g.ld_out = mixer;
        }
        SB_TRY(gemm_b16_launch(g, m->stream));
        *launches += 2;
    }
    SB_TRY(rows_mixer(m, layer, ld_u, mrows, first_pos, launches));
    SB_TRY(rows_add_contract(m, t.o, L->rattn, mrows, t.scale1, launches));
    return ff ? rows_add_contract(m, t.down, L->ract, mrows, t.scale2, launches) : STARK_B200_OK;
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
    e.x_b16 = L->f32 || L->parallel ? nullptr : static_cast<uint16_t *>(L->rh);
    e.m = mrows;
    SB_TRY(embed_norm_launch(e, s));
    const void *x = L->f32 ? static_cast<const void *>(L->rx) : L->rh;
    uint16_t *rounded = L->f32 ? nullptr : static_cast<uint16_t *>(L->rh);
    for (const Layer &layer : L->layers) {
        if (L->parallel) {
            SB_TRY(rows_parallel_layer(m, layer, mrows, first_pos, &n));
            continue;
        }
        const LayerTensors &t = tensors_of(L, layer);
        SB_TRY(rows_contract(m, t.in, x, mrows, nullptr, L->ru, L->f32 ? kGemmF32 : kGemmBf16, Gate{}, &n));
        SB_TRY(rows_mixer(m, layer, layer.mixer_width(), mrows, first_pos, &n));
        SB_TRY(rows_contract(m, t.o, L->rattn, mrows, nullptr, L->ry, kGemmF32, Gate{}, &n));
        SB_TRY(add_norm_rows_launch(L->rx, L->ry, t.norm1, mrows, L->c.width, L->c.eps, rounded, s));
        ++n;
        if (layer.d.feed_forward == STARK_B200_FF_NONE) continue;
        SB_TRY(rows_contract(m, t.gate_up, x, mrows, t.gate_up_b, L->ract, kGemmGate, layer.gate(), &n));
        SB_TRY(rows_contract(m, t.down, L->ract, mrows, t.down_b, L->ry, kGemmF32, Gate{}, &n));
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
        SB_TRY(norm_rows_launch(L->rx, L->picked, n, L->final_norm, L->c.width, L->c.eps,
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

constexpr uint32_t bit(uint32_t id) { return 1u << id; }

uint32_t model_tensors(const stark_b200_layered_config &c) {
    uint32_t want = bit(STARK_B200_LAYERED_EMBED) | bit(STARK_B200_LAYERED_FINAL_NORM);
    if (c.flags & STARK_B200_LAYERED_HAS_EMBED_NORM) want |= bit(STARK_B200_LAYERED_EMBED_NORM);
    if (!(c.flags & STARK_B200_LAYERED_TIED_HEAD)) want |= bit(STARK_B200_LAYERED_HEAD);
    if (c.bigram_buckets) want |= bit(STARK_B200_LAYERED_BIGRAM);
    return want;
}

uint32_t layer_tensors(const LayeredState *L, const Layer &l) {
    uint32_t want = bit(STARK_B200_LAYERED_NORM1) | bit(STARK_B200_LAYERED_Q) | bit(STARK_B200_LAYERED_O);
    if (l.latent()) {
        want |= bit(STARK_B200_LAYERED_DKV) | bit(STARK_B200_LAYERED_DKV_NORM) | bit(STARK_B200_LAYERED_UK) | bit(STARK_B200_LAYERED_UV);
    } else {
        want |= bit(STARK_B200_LAYERED_K) | bit(STARK_B200_LAYERED_V);
        if (l.d.conv_taps) want |= bit(STARK_B200_LAYERED_Q_CONV) | bit(STARK_B200_LAYERED_K_CONV) | bit(STARK_B200_LAYERED_V_CONV);
        if (l.d.v_mix) want |= bit(STARK_B200_LAYERED_V_SHARE);
    }
    if (L->parallel) want |= bit(STARK_B200_LAYERED_SCALE1);
    if (l.d.feed_forward == STARK_B200_FF_NONE) return want;
    want |= bit(STARK_B200_LAYERED_GATE) | bit(STARK_B200_LAYERED_UP) | bit(STARK_B200_LAYERED_DOWN);
    want |= L->parallel ? bit(STARK_B200_LAYERED_SCALE2) : bit(STARK_B200_LAYERED_NORM2);
    if (l.d.feed_forward == STARK_B200_FF_CLAMPED_GATE)
        want |= bit(STARK_B200_LAYERED_GATE_BIAS) | bit(STARK_B200_LAYERED_UP_BIAS) | bit(STARK_B200_LAYERED_DOWN_BIAS);
    return want;
}

stark_b200_status layered_ready(Model *m) {
    LayeredState *L = m->layered;
    if (L->seen != model_tensors(L->c)) return STARK_B200_INVALID_STATE;
    for (uint32_t i = 0; i < L->layers.size(); ++i)
        if (L->layers[i].tensors == i && L->layers[i].own.seen != layer_tensors(L, L->layers[i])) return STARK_B200_INVALID_STATE;
    return STARK_B200_OK;
}

// The cache alone does not describe a layer with convolutions: its recent rows are put back as they were at the start of
// the position's page, and the tokens between are run again.
stark_b200_status layered_rewind(Model *m, uint64_t position) {
    LayeredState *L = m->layered;
    if (position == m->position || position == 0) return STARK_B200_OK;
    const uint32_t page_start = (uint32_t)(position / kPageTokens * kPageTokens);
    bool any = false;
    for (const Layer &layer : L->layers) {
        if (layer.latent() || layer.taps <= 1u) continue;
        SB_TRY(short_conv_restore_launch(grouped_args(m, layer), page_start, m->stream));
        any = true;
    }
    if (!any || position == page_start) return STARK_B200_OK;
    if (!layered_rows_ready(m)) return STARK_B200_OUT_OF_MEMORY;
    return layered_rows_pass(m, L->history + page_start, (uint32_t)(position - page_start), page_start);
}

void layered_sizes(const Model *m, uint64_t *weight_bytes, uint64_t *kv_bytes_per_token) {
    const LayeredState *L = m->layered;
    const bool tied = (L->c.flags & STARK_B200_LAYERED_TIED_HEAD) != 0u;
    uint64_t w = L->head.bytes() + (tied ? 0u : (uint64_t)L->c.vocab * L->c.width * 2u) +
                 (L->c.bigram_buckets ? ((uint64_t)L->c.bigram_buckets + 1u) * L->c.width * 2u : 0u), kv = 0;
    for (const Layer &l : L->layers) {
        for (const MatrixB16 *t : {&l.own.in, &l.own.out, &l.own.uk_uv}) w += t->bytes();
        if (!L->parallel)
            for (const MatrixB16 *t : {&l.own.o, &l.own.gate_up, &l.own.down}) w += t->bytes();
        const uint64_t row = l.latent() ? l.s.row()
                                        : l.g.groups * (l.g.dim_p + l.g.vdim_p) + ((l.taps - 1u) * l.g.width() + kPageTokens - 1u) / kPageTokens;
        kv += row * (L->f32 ? 4u : 2u);
    }
    *weight_bytes = w;
    *kv_bytes_per_token = kv;
}

void layered_destroy(Model *m) {
    LayeredState *L = m->layered;
    if (!L) return;
    for (Layer &l : L->layers) {
        for (MatrixB16 *t : {&l.own.in, &l.own.out, &l.own.uk_uv}) cudaFree(t->data);
        if (!L->parallel)
            for (MatrixB16 *t : {&l.own.o, &l.own.gate_up, &l.own.down}) cudaFree(t->data);
        for (float *p : {l.own.latent_norm, l.own.norm1, l.own.norm2, l.own.gate_up_b, l.own.down_b, l.own.conv_w, l.own.scale1,
                         l.own.scale2, l.freq})
            cudaFree(p);
        for (void *p : {l.cache, l.keys, l.values, l.recent, l.tails}) cudaFree(p);
    }
    for (void *p : {(void *)L->embed, (void *)L->bigram, (void *)L->head.data, (void *)L->embed_norm, (void *)L->final_norm,
                    (void *)L->history, (void *)L->x[0], (void *)L->x[1], (void *)L->y, (void *)L->u, (void *)L->attn,
                    (void *)L->queries, (void *)L->partials, (void *)L->first_values, (void *)L->rx, (void *)L->ry, L->rh,
                    L->ru, L->rattn, L->ract, (void *)L->rq, (void *)L->rfirst, (void *)L->rgu, (void *)L->expanded,
                    (void *)L->picked, L->picked_x, (void *)L->picked_logits})
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
    f.rewind = layered_rewind;
    f.sizes = layered_sizes;
    f.destroy = layered_destroy;
    return f;
}
const ModelFamily kLayeredFamily = make_layered_family();

stark_b200_status check_layer(const stark_b200_layered_config &c, const stark_b200_layer_desc &d) {
    if (d.struct_size != sizeof(d)) return STARK_B200_ABI_MISMATCH;
    const bool latent = d.mixer == STARK_B200_MIXER_LATENT;
    if ((!latent && d.mixer != STARK_B200_MIXER_GROUPED) || d.feed_forward > STARK_B200_FF_SILU_GATE ||
        d.rot_scaling > STARK_B200_ROT_YARN ||
        (c.arrangement == STARK_B200_ARRANGE_PARALLEL && d.feed_forward == STARK_B200_FF_CLAMPED_GATE))  // has biases
        return STARK_B200_UNSUPPORTED;
    if (!d.heads || !d.dim || !d.vdim || !std::isfinite(d.scale) || (d.feed_forward != STARK_B200_FF_NONE && !d.ff_width))
        return STARK_B200_INVALID_ARGUMENT;
    if (latent &&
        (!d.kv_rank || d.rot_dim % 2u || d.rot_dims % 2u || d.rot_dims > d.rot_dim || !(d.rot_base > 0.0) ||
         (d.rot_scaling == STARK_B200_ROT_YARN && !(d.rot_factor > 0.0 && d.rot_original > 0.0 && d.rot_fast > 0.0 && d.rot_slow > 0.0))))
        return STARK_B200_INVALID_ARGUMENT;
    if (!latent && (!d.kv_heads || d.heads % d.kv_heads || !d.q_temp_every || !std::isfinite(d.q_temp_coef) || d.rot_dim))
        return STARK_B200_INVALID_ARGUMENT;
    return STARK_B200_OK;
}

stark_b200_status zeroed(void **p, size_t bytes) {
    SB_TRY(dmalloc(reinterpret_cast<uint8_t **>(p), bytes));
    SB_CUDA(cudaMemset(*p, 0, bytes ? bytes : 1u));
    return STARK_B200_OK;
}

stark_b200_status build_latent(Model *m, Layer &l) {
    LayeredState *L = m->layered;
    LatentShape &s = l.s;
    s.heads = l.d.heads, s.dim = l.d.dim, s.rot_dim = l.d.rot_dim, s.vdim = l.d.vdim, s.rank = l.d.kv_rank;
    s.dim_p = pad64(s.dim), s.rot_p = pad64(s.rot_dim), s.vdim_p = pad64(s.vdim), s.rank_p = pad64(s.rank);
    if (!latent_shape_supported(s)) return STARK_B200_UNSUPPORTED;
    std::vector<float> freq(std::max(1u, s.rot_p / 2u), 0.0f);
    rotation_table(l.d, freq, &l.rot.factor);
    SB_TRY(dmalloc(&l.freq, freq.size()));
    SB_CUDA(cudaMemcpy(l.freq, freq.data(), freq.size() * 4u, cudaMemcpyHostToDevice));
    l.rot.freq = l.freq;
    l.rot.pairs = l.d.rot_dims / 2u;
    SB_TRY(zeroed(&l.cache, (size_t)m->num_blocks * kPageTokens * s.row() * (L->f32 ? 4u : 2u)));
    L->max_expand = std::max(L->max_expand, s.heads * (s.dim_p + s.vdim_p));
    L->query_floats = std::max(L->query_floats, (size_t)kAttendRows * s.heads * s.row());
    for (uint32_t r = 1; r <= kAttendRows; ++r) {
        LatentArgs probe{};
        probe.s = s;
        probe.cache_f32 = L->f32;
        divide_cache(probe, r);
        L->partial_floats = std::max(L->partial_floats, latent_partial_floats(s, r, probe.splits * probe.cluster));
    }
    return STARK_B200_OK;
}

stark_b200_status build_grouped(Model *m, Layer &l) {
    LayeredState *L = m->layered;
    GroupedShape &s = l.g;
    s.heads = l.d.heads, s.groups = l.d.kv_heads, s.dim = l.d.dim, s.vdim = l.d.vdim;
    s.dim_p = pad64(s.dim), s.vdim_p = pad64(s.vdim);
    l.taps = std::max(1u, l.d.conv_taps);
    if (!grouped_shape_supported(s, l.taps)) return STARK_B200_UNSUPPORTED;
    if (!l.d.conv_taps && &tensors_of(L, l) == &l.own) {
        const std::vector<float> ones(s.width(), 1.0f);
        SB_TRY(dmalloc(&l.own.conv_w, ones.size()));
        SB_CUDA(cudaMemcpy(l.own.conv_w, ones.data(), ones.size() * 4u, cudaMemcpyHostToDevice));
    }
    const size_t element = L->f32 ? 4u : 2u, positions = (size_t)m->num_blocks * kPageTokens;
    SB_TRY(zeroed(&l.keys, positions * s.groups * s.dim_p * element));
    SB_TRY(zeroed(&l.values, positions * s.groups * s.vdim_p * element));
    SB_TRY(zeroed(&l.recent, (size_t)(l.taps + kConvSpare) * s.width() * element));
    SB_TRY(zeroed(&l.tails, (size_t)m->num_blocks * (l.taps - 1u) * s.width() * element));
    L->max_q = std::max(L->max_q, s.heads * s.dim_p);
    if (l.d.v_mix) {
        const uint32_t row = s.groups * s.vdim;
        if (L->max_first && row != L->max_first) return STARK_B200_INVALID_ARGUMENT;  // entries mix one by one
        l.mix = L->max_first ? kMixShare : kMixFirst;
        L->max_first = row;
    }
    L->query_floats = std::max(L->query_floats, (size_t)kAttendRows * s.heads * s.dim_p);
    for (uint32_t r = 1; r <= kAttendRows; ++r)
        L->partial_floats = std::max(L->partial_floats, span_partial_floats(s.heads, s.vdim_p, r, plain_splits(s, r)));
    L->partial_floats = std::max(L->partial_floats, span_partial_floats(s.heads, s.vdim_p, 1u, kMaxSplits));
    return STARK_B200_OK;
}

stark_b200_status build_layers(Model *m, const stark_b200_layer_desc *descs) {
    LayeredState *L = m->layered;
    L->layers.resize(L->c.layers);
    for (uint32_t i = 0; i < L->c.layers; ++i) {
        Layer &l = L->layers[i];
        l.d = descs[i];
        SB_TRY(check_layer(L->c, l.d));
        l.tensors = i;
        if (l.d.weights_of != UINT32_MAX) {
            if (l.d.weights_of >= L->c.layers || descs[l.d.weights_of].weights_of != UINT32_MAX) return STARK_B200_INVALID_ARGUMENT;
            // everything but the reference must equal the layer it points to
            stark_b200_layer_desc a = l.d, b = descs[l.d.weights_of];
            a.weights_of = b.weights_of = 0;
            if (memcmp(&a, &b, sizeof a) != 0) return STARK_B200_INVALID_ARGUMENT;
            l.tensors = l.d.weights_of;
        }
        l.ff_p = l.d.feed_forward == STARK_B200_FF_NONE ? 0u : pad64(l.d.ff_width);
        SB_TRY(l.latent() ? build_latent(m, l) : build_grouped(m, l));
        L->max_mixer = std::max(L->max_mixer, l.mixer_width());
        L->max_in = std::max(L->max_in, l.mixer_width() + (L->parallel ? 2u * l.ff_p : 0u));
        L->max_attn = std::max(L->max_attn, l.attn_width());
        L->max_ff = std::max(L->max_ff, l.ff_p);
        L->max_joint = std::max(L->max_joint, l.attn_width() + std::max(64u, l.ff_p));
    }
    for (const MatrixB16 &probe : {MatrixB16{nullptr, 1, L->width_p}, MatrixB16{nullptr, 1, L->parallel ? L->max_joint : L->max_attn},
                                   MatrixB16{nullptr, 1, std::max(64u, L->max_ff)}})
        if (!matvec_b16_supports(probe)) return STARK_B200_UNSUPPORTED;
    SB_TRY(dmalloc(&L->history, (size_t)m->num_blocks * kPageTokens + 1u));
    for (float **p : {&L->x[0], &L->x[1], &L->y}) SB_TRY(dmalloc(p, L->width_p));
    SB_TRY(dmalloc(&L->u, L->max_mixer));
    SB_TRY(dmalloc(&L->attn, L->max_joint));
    if (L->max_first) SB_TRY(dmalloc(&L->first_values, L->max_first));
    SB_TRY(dmalloc(&L->queries, L->query_floats));
    return dmalloc(&L->partials, L->partial_floats);
}

stark_b200_status layered_create(const stark_b200_layered_config &c, const stark_b200_layer_desc *descs, Model **out) {
    *out = nullptr;
    if (!c.vocab || !c.width || !c.layers || !c.context_tokens || c.width > 32768u || !(c.eps >= 0.0f) ||
        c.compute > STARK_B200_F32 || c.arrangement > STARK_B200_ARRANGE_PARALLEL || !std::isfinite(c.residual_mult) || (uint64_t)c.bigram_buckets + 1u > UINT32_MAX || c.bigram_mul_prev > UINT32_MAX ||
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
    L->parallel = c.arrangement == STARK_B200_ARRANGE_PARALLEL;
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

// Storage of the fused matrices, made when the first of their parts arrives.
stark_b200_status input_matrix(LayeredState *L, Layer &l) {
    LayerTensors &t = l.own;
    const uint32_t fused = L->parallel ? 2u * l.ff_p : 0u;
    SB_TRY(alloc_matrix(t.in, l.mixer_width() + fused, L->width_p));
    if (!l.ff_p) return STARK_B200_OK;
    if (fused) t.gate_up = t.in.row_range(l.mixer_width(), fused);
    else SB_TRY(alloc_matrix(t.gate_up, 2u * l.ff_p, L->width_p));
    return STARK_B200_OK;
}
stark_b200_status output_matrices(LayeredState *L, Layer &l) {
    LayerTensors &t = l.own;
    if (!L->parallel) {
        SB_TRY(alloc_matrix(t.o, L->width_p, l.attn_width()));
        return l.ff_p ? alloc_matrix(t.down, L->width_p, l.ff_p) : STARK_B200_OK;
    }
    SB_TRY(alloc_matrix(t.out, L->width_p, l.attn_width() + l.ff_p));
    t.o = t.out.column_range(0, l.attn_width());
    if (l.ff_p) t.down = t.out.column_range(l.attn_width(), l.ff_p);
    return STARK_B200_OK;
}

stark_b200_status set_model_tensor(LayeredState *L, uint32_t which, const uint16_t *src, uint32_t rows, uint32_t cols) {
    const auto &c = L->c;
    const bool tied = (c.flags & STARK_B200_LAYERED_TIED_HEAD) != 0u;
    const float offset = c.flags & STARK_B200_LAYERED_NORM_AROUND_ZERO ? 1.0f : 0.0f;
    auto shaped = [&](uint32_t r, uint32_t k) { return rows == r && cols == k; };
    switch (which) {
        case STARK_B200_LAYERED_EMBED_NORM:
        case STARK_B200_LAYERED_FINAL_NORM:
            if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(which == STARK_B200_LAYERED_EMBED_NORM ? &L->embed_norm : &L->final_norm, L->width_p, src, cols, offset));
            break;
        case STARK_B200_LAYERED_HEAD:
        case STARK_B200_LAYERED_EMBED:
            if (!shaped(c.vocab, c.width)) return STARK_B200_INVALID_ARGUMENT;
            if (which == STARK_B200_LAYERED_HEAD || tied) {
                SB_TRY(alloc_matrix(L->head, c.vocab, L->width_p));
                SB_TRY(place(L->head, 0, 0, src, cols, 0, 0, rows, cols));
                break;
            }
            if (!L->embed) SB_TRY(dmalloc(&L->embed, (size_t)rows * cols));
            SB_CUDA(cudaMemcpy(L->embed, src, (size_t)rows * cols * 2u, cudaMemcpyHostToDevice));
            break;
        default:
            if (!shaped(c.bigram_buckets + 1u, c.width)) return STARK_B200_INVALID_ARGUMENT;
            if (!L->bigram) SB_TRY(dmalloc(&L->bigram, (size_t)rows * cols));
            SB_CUDA(cudaMemcpy(L->bigram, src, (size_t)rows * cols * 2u, cudaMemcpyHostToDevice));
    }
    L->seen |= 1u << which;
    return STARK_B200_OK;
}

stark_b200_status layered_set(Model *m, uint32_t layer, uint32_t which, const uint16_t *src, uint32_t rows, uint32_t cols) {
    LayeredState *L = m->layered;
    if (m->finalized) return STARK_B200_INVALID_STATE;
    const auto &c = L->c;
    auto shaped = [&](uint32_t r, uint32_t k) { return rows == r && cols == k; };
    if (which <= STARK_B200_LAYERED_HEAD)
        return model_tensors(c) & bit(which) ? set_model_tensor(L, which, src, rows, cols) : STARK_B200_INVALID_ARGUMENT;
    if (layer >= L->layers.size() || which > STARK_B200_LAYERED_SCALE2) return STARK_B200_INVALID_ARGUMENT;
    Layer &l = L->layers[layer];
    // only a layer with tensors of its own, and only what its mixer, feed-forward and arrangement have
    if (l.tensors != layer || !(layer_tensors(L, l) & bit(which))) return STARK_B200_INVALID_ARGUMENT;
    const LatentShape &s = l.s;
    const GroupedShape &g = l.g;
    const float offset = c.flags & STARK_B200_LAYERED_NORM_AROUND_ZERO ? 1.0f : 0.0f;
    LayerTensors &t = l.own;
    SB_TRY(input_matrix(L, l));
    SB_TRY(output_matrices(L, l));
    // heads of `n` rows each, stored `padded` rows apart from row `first` of the input matrix on
    auto place_heads = [&](uint32_t first, uint32_t heads, uint32_t n, uint32_t padded) -> stark_b200_status {
        if (!shaped(heads * n, c.width)) return STARK_B200_INVALID_ARGUMENT;
        for (uint32_t h = 0; h < heads; ++h) SB_TRY(place(t.in, first + h * padded, 0, src, cols, h * n, 0, n, cols));
        return STARK_B200_OK;
    };
    auto place_taps = [&](uint32_t first, uint32_t heads, uint32_t n, uint32_t padded) -> stark_b200_status {
        if (!shaped(heads * n, l.taps)) return STARK_B200_INVALID_ARGUMENT;
        SB_TRY(alloc_vector(&t.conv_w, l.taps * g.width()));
        std::vector<float> w((size_t)l.taps * g.width());
        SB_CUDA(cudaMemcpy(w.data(), t.conv_w, w.size() * 4u, cudaMemcpyDeviceToHost));  // other parts may be there
        for (uint32_t r = 0; r < rows; ++r)
            for (uint32_t j = 0; j < l.taps; ++j)
                w[(size_t)j * g.width() + first + r / n * padded + r % n] = bf16_bits_to_f32(src[(size_t)r * l.taps + j]);
        SB_CUDA(cudaMemcpy(t.conv_w, w.data(), w.size() * 4u, cudaMemcpyHostToDevice));
        return STARK_B200_OK;
    };
    switch (which) {
        case STARK_B200_LAYERED_NORM1:
        case STARK_B200_LAYERED_NORM2:
            if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(which == STARK_B200_LAYERED_NORM1 ? &t.norm1 : &t.norm2, L->width_p, src, cols, offset));
            break;
        case STARK_B200_LAYERED_SCALE1:
        case STARK_B200_LAYERED_SCALE2:
            if (!shaped(1, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(put_vector(which == STARK_B200_LAYERED_SCALE1 ? &t.scale1 : &t.scale2, L->width_p, src, cols, 0.0f, c.residual_mult));
            break;
        case STARK_B200_LAYERED_Q:
            if (!l.latent()) {
                SB_TRY(place_heads(0, g.heads, g.dim, g.dim_p));
                break;
            }
            if (!shaped(s.heads * (s.dim + s.rot_dim), c.width)) return STARK_B200_INVALID_ARGUMENT;
            for (uint32_t h = 0; h < s.heads; ++h) {
                SB_TRY(place(t.in, h * s.q_head(), 0, src, cols, h * (s.dim + s.rot_dim), 0, s.dim, cols));
                if (s.rot_dim)
                    SB_TRY(place(t.in, h * s.q_head() + s.dim_p, 0, src, cols, h * (s.dim + s.rot_dim) + s.dim, 0, s.rot_dim, cols));
            }
            break;
        case STARK_B200_LAYERED_K: SB_TRY(place_heads(g.key_col(), g.groups, g.dim, g.dim_p)); break;
        case STARK_B200_LAYERED_V: SB_TRY(place_heads(g.value_col(), g.groups, g.vdim, g.vdim_p)); break;
        case STARK_B200_LAYERED_Q_CONV: SB_TRY(place_taps(0, g.heads, g.dim, g.dim_p)); break;
        case STARK_B200_LAYERED_K_CONV: SB_TRY(place_taps(g.key_col(), g.groups, g.dim, g.dim_p)); break;
        case STARK_B200_LAYERED_V_CONV: SB_TRY(place_taps(g.value_col(), g.groups, g.vdim, g.vdim_p)); break;
        case STARK_B200_LAYERED_V_SHARE:
            if (!shaped(1, 1)) return STARK_B200_INVALID_ARGUMENT;
            t.share = bf16_bits_to_f32(src[0]);
            break;
        case STARK_B200_LAYERED_DKV:
            if (!shaped(s.rank + s.rot_dim, c.width)) return STARK_B200_INVALID_ARGUMENT;
            SB_TRY(place(t.in, s.q_width(), 0, src, cols, 0, 0, s.rank, cols));
            if (s.rot_dim) SB_TRY(place(t.in, s.q_width() + s.rank_p, 0, src, cols, s.rank, 0, s.rot_dim, cols));
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
        case STARK_B200_LAYERED_O: {
            const uint32_t heads = l.d.heads, n = l.d.vdim, n_p = l.attn_width() / heads;
            if (!shaped(c.width, heads * n)) return STARK_B200_INVALID_ARGUMENT;
            for (uint32_t h = 0; h < heads; ++h) SB_TRY(place(t.o, 0, h * n_p, src, cols, 0, h * n, rows, n));
            break;
        }
        case STARK_B200_LAYERED_GATE:
        case STARK_B200_LAYERED_UP:
            if (!shaped(l.d.ff_width, c.width)) return STARK_B200_INVALID_ARGUMENT;
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
