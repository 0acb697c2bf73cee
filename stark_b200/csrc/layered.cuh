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

// A bf16 matrix [rows, cols], row-major without gaps, cols a multiple of 64.
struct MatrixB16 {
    uint16_t *data = nullptr;
    uint32_t rows = 0, cols = 0;
    size_t bytes() const { return (size_t)rows * cols * 2u; }
};

// ---- dense contractions over a bf16 matrix (dense_b16.cu, gemm_b16.cu) --------------------------------------------
// How a one-row contraction gets its input row (f32 in every case; computed by every CTA, the first one stores it).
enum RowPrologue : uint32_t {
    kRowPlain = 0,       // x
    kRowAddNorm = 1,     // x + norm(y): the residual add of a sublayer's normed output
    kRowAddNormNorm = 2  // norm(x + norm(y)): the same, then the model's last norm
};
enum RowEpilogue : uint32_t {
    kRowStore = 0,   // out = W x (+ bias)
    kRowGate = 1,    // rows are 16 gate / 16 up in turn: out = clamped_gate(W x + bias)
    kRowLogits = 2   // kRowStore plus per-CTA (maximum, first index)
};
struct MatvecArgs {
    MatrixB16 w;
    RowPrologue prologue = kRowPlain;
    RowEpilogue epilogue = kRowStore;
    const float *x = nullptr;      // [cols]
    const float *y = nullptr;      // [cols] sublayer output (kRowAddNorm*)
    const float *norm_w = nullptr; // [cols] weight around zero
    const float *last_w = nullptr; // [cols] weight around zero (kRowAddNormNorm)
    float *x_out = nullptr;        // the row behind the add, stored by the first CTA; must not alias x
    uint32_t width = 0;            // true length of the row (what the means divide by)
    float eps = 0.0f;
    const float *bias = nullptr;   // [w.rows] or nullptr
    float limit = 0.0f;            // kRowGate
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
stark_b200_status rows_gemm_f32_launch(const MatrixB16 &w, const float *x, uint32_t m, const float *bias, float *out,
                                       uint32_t ld_out, uint32_t out_cols, cudaStream_t stream);
enum GemmB16Out : uint32_t { kGemmBf16 = 0, kGemmF32 = 1, kGemmGate = 2 };
struct GemmB16Args {
    MatrixB16 w;
    const uint16_t *x;     // [x_rows, w.cols] bf16
    uint32_t x_rows, m;    // rows the buffer holds, rows in use
    uint32_t ld_x;         // elements between rows of x
    GemmB16Out kind;
    void *out;             // [m, ld_out] bf16 or f32; kGemmGate: bf16, half as many columns as w has rows
    uint32_t ld_out;
    uint32_t out_cols;     // columns stored (before the gate's halving)
    const float *bias;     // [w.rows] or nullptr
    float limit;           // kGemmGate
};
stark_b200_status gemm_b16_launch(const GemmB16Args &a, cudaStream_t stream);

// ---- row-wise operators (layered_rows.cu) -------------------------------------------------------------------------
// x = norm(table[token] * scale + bigram[hash(previous, token)]); the token's id enters the sequence's history, which is
// where the next row's previous token comes from.
struct EmbedArgs {
    const uint16_t *table, *bigram;  // bf16 [vocab, width], [buckets + 1, width]; bigram may be nullptr
    uint32_t buckets, width, vocab;
    uint64_t mul_prev, mul_cur;
    float scale, eps;
    const float *norm_w;             // [pad64(width)]
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
// x += y / rms(y) * (1 + w), rows; x_b16 (nullable) = the new x rounded
stark_b200_status add_norm_rows_launch(float *x, const float *y, const float *w, uint32_t m, uint32_t width, float eps,
                                       uint16_t *x_b16, cudaStream_t stream);
// out[i] = norm(x[rows[i]]); exactly one of out_f32 / out_b16
stark_b200_status norm_gather_rows_launch(const float *x, const uint32_t *rows, uint32_t count, const float *w,
                                          uint32_t width, float eps, float *out_f32, uint16_t *out_b16, cudaStream_t stream);
// act = clamped_gate(gu) over rows of 16 gate / 16 up values in turn, f32
stark_b200_status clamped_gate_rows_launch(const float *gu, float *act, uint32_t m, uint32_t ff_padded, float limit,
                                           cudaStream_t stream);

// ---- latent attention (latent_attention.cu, latent_attend_mma.cu, latent_attention_tc.cu) -----------------------
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
constexpr uint32_t kLatentMaxSplits = 64;
inline size_t latent_partial_floats(const LatentShape &s, uint32_t rows, uint32_t splits) {
    return (size_t)rows * s.heads * splits * (s.rank_p + 4u);
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
