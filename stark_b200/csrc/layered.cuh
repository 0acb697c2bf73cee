// Layered decoders: models whose configuration lists every layer's mixer and feed-forward with sizes of their own, over
// bf16 weights, with the residual stream, norms, angles, scores and softmax in f32.  The family behind the shared token
// loop (token_loop.cu) is layered_model.cu; its operators are declared here and take their sizes and constants as
// arguments.
//
// Sizes inside.  Every matrix is stored with its row length, its per-head blocks and its output rows padded to multiples
// of 64 by zero rows and columns, and every activation row likewise, so that the kernels and the copy engine see aligned
// blocks only, whatever the model's sizes are.  Padding contributes exact zeros; means divide by the true width.
#pragma once
#include <vector>

#include "context.cuh"
#include "ops.cuh"

namespace sb {

inline uint32_t pad64(uint32_t n) { return (n + 63u) & ~63u; }

// A bf16 matrix [rows, cols], row-major, cols a multiple of 64; ld (a multiple of 64, 0: cols) is the distance of rows, so
// that a run of columns of a stored matrix is a matrix too.
struct MatrixB16 {
    uint16_t *data = nullptr;
    uint32_t rows = 0, cols = 0, ld = 0;
    uint32_t pitch() const { return ld ? ld : cols; }
    size_t bytes() const { return (size_t)rows * cols * 2u; }
    MatrixB16 row_range(uint32_t first, uint32_t n) const { return {data + (size_t)first * pitch(), n, cols, pitch()}; }
    MatrixB16 column_range(uint32_t first, uint32_t n) const { return {data + first, rows, n, pitch()}; }
};

// The gated unit of a feed-forward: what becomes of a gate value and an up value.
enum GateKind : uint32_t {
    kGateClamped = 0,  // clamped halves, up half around one
    kGateSilu = 1      // silu(g) * u
};
struct Gate {
    GateKind kind = kGateClamped;
    float limit = 0.0f;  // kGateClamped
};

// ---- dense contractions over a bf16 matrix (dense_b16.cu, gemm_b16.cu) --------------------------------------------
// How a one-row contraction gets its input row (f32 in every case; computed by every CTA, the first one stores it).
enum RowPrologue : uint32_t {
    kRowPlain = 0,       // x
    kRowAddNorm = 1,     // x + norm(y): the residual add of a sublayer's normed output
    kRowAddNormNorm = 2, // norm(x + norm(y)): the same, then the model's last norm
    kRowNorm = 3         // norm(x)
};
enum RowEpilogue : uint32_t {
    kRowStore = 0,   // out = W x (+ bias)
    kRowGate = 1,    // rows behind stored_rows are 16 gate / 16 up in turn: out = gate(W x + bias)
    kRowLogits = 2,  // kRowStore plus per-CTA (maximum, first index)
    kRowResidual = 3 // out = residual + scale_a * (W x over the first split_col columns) + scale_b * (over the others)
};
struct MatvecArgs {
    MatrixB16 w;
    RowPrologue prologue = kRowPlain;
    RowEpilogue epilogue = kRowStore;
    const float *x = nullptr;      // [cols]
    const float *y = nullptr;      // [cols] sublayer output (kRowAddNorm*)
    const float *norm_w = nullptr; // [cols]
    const float *last_w = nullptr; // [cols] (kRowAddNormNorm)
    float *x_out = nullptr;        // the row behind the add, stored by the first CTA; must not alias x
    uint32_t width = 0;            // true length of the row (what the means divide by)
    float eps = 0.0f;
    const float *bias = nullptr;   // [w.rows] or nullptr
    Gate gate;                     // kRowGate
    uint32_t stored_rows = 0;      // kRowGate: rows (a multiple of 32) in front of the gated ones, stored plainly
    float *stored_out = nullptr;
    const float *residual = nullptr, *scale_a = nullptr, *scale_b = nullptr;  // [w.rows]; kRowResidual (out may be residual)
    uint32_t split_col = 0;        // kRowResidual: a multiple of 8
    float *out = nullptr;
    uint32_t out_rows = 0;         // rows of w that are stored (kRowLogits: the vocabulary)
    float *partial_max = nullptr;
    uint32_t *partial_index = nullptr;
    uint32_t *out_grid = nullptr;  // host: CTAs launched (= partials written)
    bool pdl = false;
};
bool matvec_b16_supports(const MatrixB16 &w);
stark_b200_status matvec_b16_launch(const MatvecArgs &a, cudaStream_t stream);

// y[m, n] = x[m, k] w[n, k]^T (+ bias), everything f32 on the CUDA cores: the exact form of a several-rows contraction.
// With add_scale: y += add_scale[n] * (x w^T).
stark_b200_status rows_gemm_f32_launch(const MatrixB16 &w, const float *x, uint32_t m, const float *bias, float *out,
                                       uint32_t ld_out, uint32_t out_cols, cudaStream_t stream, const float *add_scale = nullptr);
enum GemmB16Out : uint32_t { kGemmBf16 = 0, kGemmF32 = 1, kGemmGate = 2, kGemmResidual = 3 };
struct GemmB16Args {
    MatrixB16 w;
    const uint16_t *x;     // [x_rows, w.cols] bf16
    uint32_t x_rows, m;    // rows the buffer holds, rows in use
    uint32_t ld_x;         // elements between rows of x
    GemmB16Out kind;
    void *out;             // [m, ld_out] bf16 or f32; kGemmGate: bf16, half as many columns as w has gated rows
    uint32_t ld_out;
    uint32_t out_cols;     // columns stored (before the gate's halving)
    const float *bias;     // [w.rows] or nullptr
    Gate gate;             // kGemmGate
    uint32_t stored_cols;  // kGemmGate: columns (a multiple of 32) in front of the gated ones, stored plainly as bf16
    uint16_t *stored_out;  // [m, ld_stored]
    uint32_t ld_stored;
    const float *scale;    // [w.rows]; kGemmResidual: out (f32) += scale * product
};
stark_b200_status gemm_b16_launch(const GemmB16Args &a, cudaStream_t stream);

// ---- row-wise operators (layered_rows.cu) -------------------------------------------------------------------------
// x = norm(table[token] * scale + bigram[hash(previous, token)]); the token's id enters the sequence's history, which is
// where the next row's previous token comes from.  norm_w == nullptr: no norm.  Norm weights multiply as they are here and
// below (a design whose stored weights lie around zero has one added when they are loaded).
struct EmbedArgs {
    const uint16_t *table, *bigram;  // bf16 [vocab, ld_table], [buckets + 1, width]; bigram may be nullptr
    uint32_t ld_table;
    uint32_t buckets, width, vocab;
    uint64_t mul_prev, mul_cur;
    float scale, eps;
    const float *norm_w;             // [pad64(width)] or nullptr
    const uint32_t *tokens;          // a pass: ids of its rows; nullptr: one row, token and position from `state`
    uint32_t first_pos;
    const StepState *state;
    uint32_t *history;               // [context] ids by position
    float *x;                        // [m, pad64(width)]
    uint16_t *x_b16;                 // the same rounded, or nullptr
    uint32_t m;
    bool pdl;
};
stark_b200_status embed_norm_launch(const EmbedArgs &a, cudaStream_t stream);
// x += y / rms(y) * w, rows; x_b16 (nullable) = the new x rounded
stark_b200_status add_norm_rows_launch(float *x, const float *y, const float *w, uint32_t m, uint32_t width, float eps,
                                       uint16_t *x_b16, cudaStream_t stream);
// out[i] = norm(x[rows ? rows[i] : i]); exactly one of out_f32 / out_b16
stark_b200_status norm_rows_launch(const float *x, const uint32_t *rows, uint32_t count, const float *w, uint32_t width,
                                   float eps, float *out_f32, uint16_t *out_b16, cudaStream_t stream);
// act = gate(gu) over rows (ld_gu apart) of 16 gate / 16 up values in turn, f32
stark_b200_status gate_rows_launch(const float *gu, uint32_t ld_gu, float *act, uint32_t m, uint32_t ff_padded, Gate gate,
                                   cudaStream_t stream);

// ---- attention over spans of a paged cache on the CUDA cores (span_attend.cu): any sizes, f32 or bf16 cache ----------
// Keys of key head g on page p: rows of key_pitch values at keys + ((block_table[p] * key_heads + g) * kPageTokens) *
// key_pitch, values likewise; query head h uses key head h / (heads / key_heads).
struct SpanAttendArgs {
    const float *queries;      // [m, heads, width], scaled by scale * log2(e)
    uint32_t heads, key_heads, width, out_width;
    const void *keys, *values;
    uint32_t key_pitch, value_pitch;
    bool cache_f32;
    const int32_t *block_table;
    const StepState *state;    // one row: its position is read on the device; nullptr: rows at first_pos + i
    uint32_t first_pos, m, splits;
    float *partials;           // [m, heads, splits, out_width + 4]: maximum, sum, -, -, weighted values
    void *out;                 // span_merge: [m, ld_out], head h at h * out_width
    uint32_t ld_out;
    bool out_b16, pdl;
};
constexpr uint32_t kMaxSplits = 64;
bool span_attend_supports(uint32_t width, uint32_t out_width);
inline size_t span_partial_floats(uint32_t heads, uint32_t out_width, uint32_t rows, uint32_t splits) {
    return (size_t)rows * heads * splits * (out_width + 4u);
}
stark_b200_status span_attend_launch(const SpanAttendArgs &a, cudaStream_t stream);
// out = sum over the spans of their weighted values / sum of their sums
stark_b200_status span_merge_launch(const SpanAttendArgs &a, cudaStream_t stream);

// ---- causal attention of a prompt pass on the tensor cores (layered_attention_tc.cu) ----------------------------------
// Query rows are [m, heads * key width] bf16 (whole blocks of 64 a head).  The key tile of a page is put together from
// own_blocks blocks of 64 columns out of `keys` (head h: columns h * key_stride ...) and shared_blocks out of `shared`
// (every head the same); values come from `values`.  A page's rows for key head g start at (block_table[p] * key_heads + g)
// * 64 in keys and values; query head h uses key head h / (heads / key_heads).
struct AttendTile {
    const uint16_t *base;
    uint32_t columns, rows, ld;  // what the copy engine may touch
    uint32_t first, stride;      // column of head 0, columns from a head to the next
};
struct AttendTcArgs {
    const uint16_t *queries;
    uint32_t ld_q, heads, key_heads;
    AttendTile keys, values, shared;   // shared: first = column, stride 0
    uint32_t own_blocks, shared_blocks, value_blocks;
    const int32_t *block_table;
    uint32_t first_pos, m;
    float scale;                       // positive
    // A bound on |query . key| known without looking: dim_bound * |1 + temp_coef * ln((position + 1) / temp_every + 1)|.
    // Where it is small enough it stands in for the row's maximum and the keys are walked once.  0: not known.
    float dim_bound, temp_coef;
    uint32_t temp_every;
    uint16_t *out;                     // [m, heads * value_blocks * 64]
    uint32_t *error_word;
};
bool attend_tc_supports(uint32_t key_blocks, uint32_t value_blocks);
stark_b200_status attend_tc_launch(const AttendTcArgs &a, cudaStream_t stream);

// ---- grouped-query attention with short convolutions (grouped_attention.cu, grouped_attend_mma.cu) --------------------
// The projected row of a position is u = [queries, heads x dim_p | keys, groups x dim_p | values, groups x vdim_p].  Each
// of its channels goes through a causal convolution over time; queries and keys are divided by their root mean square per
// head, queries are multiplied by a temperature of their position, values may be mixed with those of the first layer that
// mixes.  Keys and values are cached per page and head, [page][group][64][dim_p] and [page][group][64][vdim_p].
// State of the convolutions beside the cache: the last projected rows by position modulo recent_rows(), and per page the
// rows of its last taps - 1 positions, from which a rewind to the next page's start continues.
struct GroupedShape {
    uint32_t heads, groups, dim, vdim;  // true sizes
    uint32_t dim_p, vdim_p;             // padded to 64
    __host__ __device__ uint32_t per() const { return heads / groups; }
    __host__ __device__ uint32_t key_col() const { return heads * dim_p; }
    __host__ __device__ uint32_t value_col() const { return key_col() + groups * dim_p; }
    __host__ __device__ uint32_t width() const { return value_col() + groups * vdim_p; }
};
constexpr uint32_t kConvSpare = 16;  // rows of a pass that can enter the recent rows while its first rows still read them
struct ShortConv {
    const float *w;      // [taps][width()]
    uint32_t taps;
    void *recent;        // [taps + kConvSpare][width()], bf16 or f32 as the cache
    void *tails;         // [pages][taps - 1][width()]
    __host__ __device__ uint32_t recent_rows() const { return taps + kConvSpare; }
};
enum ValueMix : uint32_t { kMixNone = 0, kMixFirst = 1, kMixShare = 2 };
struct GroupedArgs {
    GroupedShape s;
    ShortConv conv;
    const void *u;             // [m, ld_u] projected rows, f32 (or bf16: u_b16)
    bool u_b16;
    uint32_t ld_u;
    float eps, scale, temp_coef;
    uint32_t temp_every;
    ValueMix mix;
    float share;               // kMixShare
    float *first_values;       // [m, groups * vdim]: written by kMixFirst, read by kMixShare
    void *keys, *values;
    bool cache_f32;
    const int32_t *block_table;
    uint32_t num_blocks;
    const StepState *state;    // one row: its position is read on the device; nullptr: rows at first_pos + i
    uint32_t first_pos, m;
    float *queries;            // grouped_rows: [m, heads, dim_p] scaled by scale * log2(e) ...
    uint16_t *queries_b16;     // ... or unscaled, rounded
    float *partials;           // grouped_attend_mma: [heads, splits, vdim_p + 4] where splits > 1
    uint32_t splits, cluster;  // partials per head; spans of the cache merged into each (1, 2, 4 or 8)
    uint32_t beside_smem;      // grouped_attend_mma: shared memory of an SM it leaves for the CTAs of the kernels around it
    float *out;                // grouped_attend_mma: [heads * vdim_p] where splits == 1
    uint32_t *error_word;
    bool pdl;
};
bool grouped_shape_supported(const GroupedShape &s, uint32_t taps);
// Convolutions, norms, temperature and mixing of m rows; keys and values into the cache, the convolutions' state kept.
stark_b200_status grouped_rows_launch(const GroupedArgs &a, cudaStream_t stream);
// One token: the same and its attention in one launch, over a bf16 cache on the tensor cores.
constexpr uint32_t kGroupedHeadTile = 8;  // query heads of a key / value head a CTA takes there
bool grouped_attend_mma_supports(const GroupedShape &s);
stark_b200_status grouped_attend_mma_launch(const GroupedArgs &a, cudaStream_t stream);
// The recent rows as they were before position `position` (a page's start), from the page tails.
stark_b200_status short_conv_restore_launch(const GroupedArgs &a, uint32_t position, cudaStream_t stream);

// ---- latent attention (latent_attention.cu, latent_attend_mma.cu, layered_attention_tc.cu) ----------------------
// Cache of one layer: pages of kPageTokens rows of [latent, padded | rotated key part, padded], bf16 or f32.
struct LatentShape {
    uint32_t heads, dim, rot_dim, vdim, rank;       // true sizes
    uint32_t dim_p, rot_p, vdim_p, rank_p;          // padded to 64
    __host__ __device__ uint32_t q_head() const { return dim_p + rot_p; }
    __host__ __device__ uint32_t q_width() const { return heads * q_head(); }
    __host__ __device__ uint32_t row() const { return rank_p + rot_p; }  // cache row = output row of the down projection behind the queries
};
struct Rotation {
    const float *freq;   // [rot_p / 2] angle per position of pair i (device); pairs past `pairs` pass unchanged
    uint32_t pairs;
    float factor;        // on cos and sin
};
struct LatentArgs {
    LatentShape s;
    Rotation rot;
    const void *qd;            // rows [queries | latent, key part] of the fused projection, f32 (or bf16: qd_b16)
    bool qd_b16;
    uint32_t ld_qd;
    const float *latent_norm;  // [rank_p], plain weight
    float eps, scale;
    MatrixB16 uk_uv;           // [heads * dim_p + heads * vdim_p, rank_p]
    void *cache;
    bool cache_f32;
    const int32_t *block_table;
    uint32_t num_blocks;
    const StepState *state;    // one row: its position is read on the device; nullptr: rows at first_pos + i
    uint32_t first_pos, m;
    // absorbed form
    float *queries;            // [m, heads, row()] scaled by scale * log2(e)
    float *partials;           // [m, heads, splits, rank_p + 4]
    uint32_t splits, cluster;  // partials per head; spans of the cache merged into each before it is written (1..8)
    // expanded form (prompt passes)
    uint16_t *expanded;        // [pages * 64, heads * (dim_p + vdim_p)]
    void *out;                 // [m, heads * vdim_p] f32, or bf16 (out_b16)
    bool out_b16;
    uint32_t *error_word;
    bool pdl;
};
inline size_t latent_partial_floats(const LatentShape &s, uint32_t rows, uint32_t splits) {
    return span_partial_floats(s.heads, s.rank_p, rows, splits);
}
bool latent_shape_supported(const LatentShape &s);
// The absorbed form, three launches: queries into the latent space (and the new rows into the cache), attention over
// the cached rows in spans, merge of the spans and values out of the latent space.
stark_b200_status latent_query_launch(const LatentArgs &a, cudaStream_t stream);
stark_b200_status latent_attend_launch(const LatentArgs &a, cudaStream_t stream);
stark_b200_status latent_value_launch(const LatentArgs &a, cudaStream_t stream);
// latent_attend on the tensor cores over a bf16 cache (latent_attend_mma.cu): what latent_attend_launch calls when the
// shape allows it.
bool latent_attend_mma_supports(const LatentShape &s);
stark_b200_status latent_attend_mma_launch(const LatentArgs &a, cudaStream_t stream);
// The expanded form for prompt passes: new rows into the cache and the queries' rotation in place (bf16 rows), keys and
// values of every visible row by one contraction, causal attention on the tensor cores.
bool latent_prefill_tc_supports(const LatentShape &s);
stark_b200_status latent_rotate_append_launch(const LatentArgs &a, cudaStream_t stream);
stark_b200_status latent_prefill_tc_launch(const LatentArgs &a, cudaStream_t stream);

}  // namespace sb
