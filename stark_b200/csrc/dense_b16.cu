// One-row contractions over bf16 matrices (the decode path of the layered decoders) and the f32 several-rows form.
//
// y = W x is bound by the bytes of W.  A CTA's warps each take pairs of rows (the gate and the up row of one unit, or
// two neighbours) and stream them with eight 16-byte loads in flight per lane; two 256-thread CTAs per SM keep 64 KB
// in flight.  The first batch of loads is issued before the wait on the previous kernel: weights depend on nothing.
// Where there are too few pairs for the SMs' warps, several warps of a CTA share a pair, each taking its batches of columns.
// The input row stays f32 throughout (a bf16 weight times an f32 activation, f32 accumulation), so the one-row path has
// no rounding of activations at all and serves the 32-bit mode unchanged.
// The input row is formed by every CTA in its prologue: plain, its norm, or the residual add of a normed sublayer output,
// or that followed by the model's last norm.  Rows in front of gated ones may be stored plainly (one pass over the row for
// a mixer's projections and a feed-forward's gate and up halves), and two contractions that end in the same residual add
// may share a launch, their inputs and weights side by side (kRowResidual).
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kWarps = 8, kThreads = kWarps * 32u;
constexpr uint32_t kChunk = 256;   // elements of a row one warp load covers: 32 lanes x 8
constexpr uint32_t kUnroll = 4;    // chunks of two rows in flight: 8 loads of 16 bytes per lane

// Where element e of the input row sits in shared memory: within a chunk of 256, the first four values of all lanes and
// then the second four, so that a lane's two 16-byte reads are conflict-free across the warp.
__device__ inline uint32_t spread(uint32_t e) {
    const uint32_t in = e & 255u;
    return (e & ~255u) + ((in & 4u) << 5) + ((in >> 3) << 2) + (in & 3u);
}

__device__ inline void fma8(float &acc, const uint4 &w, const float4 &a, const float4 &b) {
    acc = fmaf(__uint_as_float(w.x << 16), a.x, acc);
    acc = fmaf(__uint_as_float(w.x & 0xffff0000u), a.y, acc);
    acc = fmaf(__uint_as_float(w.y << 16), a.z, acc);
    acc = fmaf(__uint_as_float(w.y & 0xffff0000u), a.w, acc);
    acc = fmaf(__uint_as_float(w.z << 16), b.x, acc);
    acc = fmaf(__uint_as_float(w.z & 0xffff0000u), b.y, acc);
    acc = fmaf(__uint_as_float(w.w << 16), b.z, acc);
    acc = fmaf(__uint_as_float(w.w & 0xffff0000u), b.w, acc);
}

struct MatvecParams {
    const uint16_t *w;
    uint32_t rows, cols;  // rows of w are cols apart
    const float *x, *y, *norm_w, *last_w;
    float *x_out;
    uint32_t width;
    float eps;
    const float *bias;
    Gate gate;
    float *out;
    uint32_t out_rows;
    float *partial_max;
    uint32_t *partial_index;
    uint32_t pairs;         // row pairs
    uint32_t stored_pairs;  // kRowGate: pairs of neighbours in front of the gated pairs
    float *stored_out;
    const float *residual, *scale_a, *scale_b;
    uint32_t split_col;
    uint32_t share;         // warps of a CTA that share a pair: 1, 2, 4 or 8
};

template <uint32_t PRO, uint32_t EPI>
__global__ void __launch_bounds__(kThreads, 2) matvec_b16_kernel(const MatvecParams p) {
    extern __shared__ __align__(16) float xs[];  // [cols rounded up to 256]
    __shared__ float scratch[32];
    __shared__ float best_v[kWarps];
    __shared__ uint32_t best_i[kWarps];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    const uint32_t chunks = (p.cols + kChunk - 1u) / kChunk;
    __shared__ float parts[2][kWarps][4];  // of a shared pair's sums
    const uint32_t share = EPI == kRowLogits ? 1u : p.share, slot = warp / share, sub = warp % share, per_cta = kWarps / share;
    const uint32_t stride = gridDim.x * per_cta, first_chunk = sub * kUnroll;
    uint32_t pair = blockIdx.x * per_cta + slot;

    // rows of a pair: gate and up 16 apart, or neighbours
    auto is_gate = [&](uint32_t pr) { return EPI == kRowGate && pr >= p.stored_pairs; };
    auto row0 = [&](uint32_t pr) {
        if (!is_gate(pr)) return 2u * pr;
        const uint32_t unit = pr - p.stored_pairs;
        return 2u * p.stored_pairs + (unit >> 4) * 32u + (unit & 15u);
    };
    auto apart = [&](uint32_t pr) { return is_gate(pr) ? 16u : 1u; };
    uint4 buf[2][kUnroll][2];
    auto fetch = [&](uint4 (&b)[kUnroll][2], uint32_t pr, uint32_t chunk) {
        const uint32_t r = row0(pr), step = apart(pr);
#pragma unroll
        for (uint32_t u = 0; u < kUnroll; ++u) {
            const uint32_t col = (chunk + u) * kChunk + lane * 8u;
            const bool in = pr < p.pairs && col < p.cols;
#pragma unroll
            for (uint32_t j = 0; j < 2u; ++j) {
                const uint32_t rr = r + j * step;
                b[u][j] = in && rr < p.rows ? ldg_nc_v4(p.w + (size_t)rr * p.cols + col) : make_uint4(0u, 0u, 0u, 0u);
            }
        }
    };
    fetch(buf[0], pair, first_chunk);

    pdl_launch_dependents();
    pdl_wait();
    // ---- the input row
    const uint32_t padded = chunks * kChunk;
    if (PRO == kRowPlain) {
        for (uint32_t i = threadIdx.x * 4u; i < padded; i += kThreads * 4u) {
            const float4 v = i < p.cols ? *reinterpret_cast<const float4 *>(p.x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            *reinterpret_cast<float4 *>(xs + spread(i)) = v;
        }
    } else if (PRO == kRowNorm) {
        float s = 0.0f;
        for (uint32_t i = threadIdx.x * 4u; i < padded; i += kThreads * 4u) {
            const float4 v = i < p.cols ? *reinterpret_cast<const float4 *>(p.x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            *reinterpret_cast<float4 *>(xs + spread(i)) = v;
        }
        const float inv = inverse_rms(block_sum(s, scratch), p.width, p.eps);
        for (uint32_t i = threadIdx.x * 4u; i < p.cols; i += kThreads * 4u) {  // each thread its own elements
            float4 v = *reinterpret_cast<float4 *>(xs + spread(i));
            const float4 g = *reinterpret_cast<const float4 *>(p.norm_w + i);
            v.x *= inv * g.x, v.y *= inv * g.y, v.z *= inv * g.z, v.w *= inv * g.w;
            *reinterpret_cast<float4 *>(xs + spread(i)) = v;
        }
    } else {
        float s = 0.0f;
        for (uint32_t i = threadIdx.x * 4u; i < padded; i += kThreads * 4u) {
            const float4 v = i < p.cols ? *reinterpret_cast<const float4 *>(p.y + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            *reinterpret_cast<float4 *>(xs + spread(i)) = v;
        }
        float inv = inverse_rms(block_sum(s, scratch), p.width, p.eps);
        s = 0.0f;
        for (uint32_t i = threadIdx.x * 4u; i < p.cols; i += kThreads * 4u) {  // each thread its own elements
            float4 v = *reinterpret_cast<float4 *>(xs + spread(i));
            const float4 x = *reinterpret_cast<const float4 *>(p.x + i), g = *reinterpret_cast<const float4 *>(p.norm_w + i);
            v.x = x.x + v.x * inv * g.x;
            v.y = x.y + v.y * inv * g.y;
            v.z = x.z + v.z * inv * g.z;
            v.w = x.w + v.w * inv * g.w;
            *reinterpret_cast<float4 *>(xs + spread(i)) = v;
            if (blockIdx.x == 0 && p.x_out) *reinterpret_cast<float4 *>(p.x_out + i) = v;
            s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        if (PRO == kRowAddNormNorm) {
            inv = inverse_rms(block_sum(s, scratch), p.width, p.eps);
            for (uint32_t i = threadIdx.x * 4u; i < p.cols; i += kThreads * 4u) {
                float4 v = *reinterpret_cast<float4 *>(xs + spread(i));
                const float4 g = *reinterpret_cast<const float4 *>(p.last_w + i);
                v.x *= inv * g.x, v.y *= inv * g.y, v.z *= inv * g.z, v.w *= inv * g.w;
                *reinterpret_cast<float4 *>(xs + spread(i)) = v;
            }
        }
    }
    __syncthreads();

    float top = -INFINITY;
    uint32_t top_i = 0xffffffffu;
    bool bad = false;
    uint32_t chunk = first_chunk, cur = 0, turn = 0;
    const uint32_t lead = share > 1u ? slot : 0u;  // warps that share pairs go on until the CTA's first one has none
    float acc[2] = {0.0f, 0.0f}, behind[2] = {0.0f, 0.0f};  // behind: columns from split_col on
    float res[2], sa[2], sb[2];
    auto fetch_residual = [&](uint32_t pr) {  // asked for when a pair begins, used when it ends
        if constexpr (EPI == kRowResidual) {
#pragma unroll
            for (uint32_t j = 0; j < 2u; ++j) {
                const uint32_t r = 2u * pr + j;
                const bool in = pr < p.pairs && r < p.out_rows;
                res[j] = in ? p.residual[r] : 0.0f;
                sa[j] = in ? p.scale_a[r] : 0.0f;
                sb[j] = in && p.scale_b ? p.scale_b[r] : 0.0f;
            }
        }
    };
    fetch_residual(pair);
    while (pair - lead < p.pairs) {
        uint32_t next_pair = pair, next_chunk = chunk + kUnroll * share;
        if (next_chunk >= chunks) next_chunk = first_chunk, next_pair = pair + stride;
        auto consume = [&](uint4 (&now)[kUnroll][2], uint4 (&then)[kUnroll][2]) {
            fetch(then, next_pair, next_chunk);
#pragma unroll
            for (uint32_t u = 0; u < kUnroll; ++u) {
                if (chunk + u >= chunks) break;
                const float *xc = xs + (chunk + u) * kChunk + lane * 4u;
                const float4 a = *reinterpret_cast<const float4 *>(xc), b = *reinterpret_cast<const float4 *>(xc + 128);
                if (EPI == kRowResidual) {
                    const bool first = (chunk + u) * kChunk + lane * 8u < p.split_col;
#pragma unroll
                    for (uint32_t j = 0; j < 2u; ++j) {
                        float dot = 0.0f;
                        fma8(dot, now[u][j], a, b);
                        acc[j] += first ? dot : 0.0f;
                        behind[j] += first ? 0.0f : dot;
                    }
                } else {
                    fma8(acc[0], now[u][0], a, b);
                    fma8(acc[1], now[u][1], a, b);
                }
            }
        };
        if (cur == 0u) consume(buf[0], buf[1]);
        else consume(buf[1], buf[0]);
        cur ^= 1u;
        if (next_pair != pair) {
            float v0 = warp_sum(acc[0]), v1 = warp_sum(acc[1]);
            acc[0] = acc[1] = 0.0f;
            float w0 = 0.0f, w1 = 0.0f;
            if constexpr (EPI == kRowResidual) {
                w0 = warp_sum(behind[0]), w1 = warp_sum(behind[1]);
                behind[0] = behind[1] = 0.0f;
            }
            if (EPI != kRowLogits && share > 1u) {  // the same number of times in every warp
                float *mine = parts[turn][warp];
                if (lane == 0) mine[0] = v0, mine[1] = v1, mine[2] = w0, mine[3] = w1;
                __syncthreads();
                for (uint32_t i = 1; i < share; ++i) {  // the first of the sharing warps has the sum
                    const float *other = parts[turn][slot * share + i];
                    v0 += other[0], v1 += other[1], w0 += other[2], w1 += other[3];
                }
                turn ^= 1u;
            }
            if constexpr (EPI == kRowResidual) {
                v0 = fmaf(sb[0], w0, fmaf(sa[0], v0, res[0]));
                v1 = fmaf(sb[1], w1, fmaf(sa[1], v1, res[1]));
                fetch_residual(next_pair);
            }
            if (lane == 0 && sub == 0u && pair < p.pairs) {
                const uint32_t r = row0(pair), step = apart(pair);
                if (p.bias) v0 += p.bias[r], v1 += r + step < p.rows ? p.bias[r + step] : 0.0f;
                if (is_gate(pair)) {
                    p.out[pair - p.stored_pairs] = gated(p.gate, v0, v1);
                } else if (EPI == kRowGate) {
                    p.stored_out[r] = v0;
                    p.stored_out[r + 1u] = v1;
                } else {
                    if (r < p.out_rows) p.out[r] = v0;
                    if (r + 1u < p.out_rows) p.out[r + 1u] = v1;
                    if (EPI == kRowLogits) {
                        bad |= r < p.out_rows && !isfinite(v0);
                        bad |= r + 1u < p.out_rows && !isfinite(v1);
                        if (r < p.out_rows && v0 > top) top = v0, top_i = r;
                        if (r + 1u < p.out_rows && v1 > top) top = v1, top_i = r + 1u;
                    }
                }
            }
        }
        pair = next_pair;
        chunk = next_chunk;
    }
    if (EPI == kRowLogits) {
        // a row with a logit that is not finite has no greedy pick: an infinite maximum says so to the final reduction
        if (lane == 0) best_v[warp] = bad ? INFINITY : top, best_i[warp] = bad ? 0u : top_i;
        __syncthreads();
        if (threadIdx.x == 0) {
            top = best_v[0], top_i = best_i[0];
            for (uint32_t w = 1; w < kWarps; ++w)
                if (best_v[w] > top || (best_v[w] == top && best_i[w] < top_i)) top = best_v[w], top_i = best_i[w];
            p.partial_max[blockIdx.x] = top;
            p.partial_index[blockIdx.x] = top_i;
        }
    }
}

// 64 x 64 tile, 256 threads of 4 x 4 outputs, K in steps of 32
constexpr uint32_t kTile = 64, kStepK = 32;
__global__ void __launch_bounds__(256) rows_gemm_f32_kernel(const uint16_t *w, uint32_t n, uint32_t k, uint32_t ld_w, const float *x,
                                                            uint32_t m, const float *bias, float *out, uint32_t ld_out,
                                                            uint32_t out_cols, const float *add_scale) {
    __shared__ float xt[kStepK][kTile + 4], wt[kStepK][kTile + 4];
    const uint32_t n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile, t = threadIdx.x;
    const uint32_t tm = (t >> 4) * 4u, tn = (t & 15u) * 4u;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < k; k0 += kStepK) {
        for (uint32_t i = t; i < kTile * kStepK; i += 256u) {
            const uint32_t r = i / kStepK, c = i % kStepK;
            xt[c][r] = m0 + r < m ? x[(size_t)(m0 + r) * k + k0 + c] : 0.0f;
            wt[c][r] = n0 + r < n ? bf16_bits_to_f32(w[(size_t)(n0 + r) * ld_w + k0 + c]) : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (uint32_t c = 0; c < kStepK; ++c) {
            const float4 a = *reinterpret_cast<const float4 *>(&xt[c][tm]), b = *reinterpret_cast<const float4 *>(&wt[c][tn]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (uint32_t i = 0; i < 4u; ++i)
        for (uint32_t j = 0; j < 4u; ++j) {
            const uint32_t r = m0 + tm + i, c = n0 + tn + j;
            if (r >= m || c >= out_cols) continue;
            float *dst = out + (size_t)r * ld_out + c;
            const float v = acc[i][j] + (bias ? bias[c] : 0.0f);
            *dst = add_scale ? fmaf(add_scale[c], v, *dst) : v;
        }
}

using MatvecKernel = void (*)(MatvecParams);
template <uint32_t PRO>
MatvecKernel pick(RowEpilogue e) {
    switch (e) {
        case kRowStore: return matvec_b16_kernel<PRO, kRowStore>;
        case kRowGate: return matvec_b16_kernel<PRO, kRowGate>;
        case kRowLogits: return matvec_b16_kernel<PRO, kRowLogits>;
        default: return PRO == kRowPlain ? matvec_b16_kernel<kRowPlain, kRowResidual> : nullptr;
    }
}

uint32_t matvec_smem(const MatrixB16 &w) { return (w.cols + kChunk - 1u) / kChunk * kChunk * 4u; }

}  // namespace

bool matvec_b16_supports(const MatrixB16 &w) { return w.cols != 0 && w.cols % 64u == 0 && matvec_smem(w) <= 200u * 1024u; }

stark_b200_status matvec_b16_launch(const MatvecArgs &a, cudaStream_t stream) {
    if (!a.w.data || !a.x || !a.out || !matvec_b16_supports(a.w) || a.w.pitch() != a.w.cols) return STARK_B200_INVALID_ARGUMENT;
    const bool adds = a.prologue == kRowAddNorm || a.prologue == kRowAddNormNorm;
    if ((adds && (!a.y || a.x_out == a.x)) || (a.prologue != kRowPlain && !a.norm_w)) return STARK_B200_INVALID_ARGUMENT;
    if (a.prologue == kRowAddNormNorm && !a.last_w) return STARK_B200_INVALID_ARGUMENT;
    if (a.epilogue == kRowLogits && (!a.partial_max || !a.partial_index)) return STARK_B200_INVALID_ARGUMENT;
    if (a.epilogue == kRowGate &&
        (a.w.rows % 32u || a.stored_rows % 32u || a.stored_rows > a.w.rows || (a.stored_rows && !a.stored_out)))
        return STARK_B200_INVALID_ARGUMENT;
    if (a.epilogue == kRowResidual &&
        (a.prologue != kRowPlain || !a.residual || !a.scale_a || a.split_col % 8u || (a.split_col < a.w.cols && !a.scale_b) ||
         a.out_rows > a.w.rows))
        return STARK_B200_INVALID_ARGUMENT;
    MatvecParams p{};
    p.w = a.w.data, p.rows = a.w.rows, p.cols = a.w.cols;
    p.x = a.x, p.y = a.y, p.norm_w = a.norm_w, p.last_w = a.last_w, p.x_out = a.x_out;
    p.width = a.width, p.eps = a.eps, p.bias = a.bias, p.gate = a.gate;
    p.out = a.out, p.out_rows = a.out_rows, p.partial_max = a.partial_max, p.partial_index = a.partial_index;
    p.pairs = (a.w.rows + 1u) / 2u;
    p.stored_pairs = a.epilogue == kRowGate ? a.stored_rows / 2u : 0u, p.stored_out = a.stored_out;
    p.residual = a.residual, p.scale_a = a.scale_a, p.scale_b = a.scale_b, p.split_col = a.split_col;
    const uint32_t smem = matvec_smem(a.w);
    const uint32_t most = 148u * (smem <= 100u * 1024u ? 2u : 1u), batches = (a.w.cols + kChunk * kUnroll - 1u) / (kChunk * kUnroll);
    p.share = 1;
    while (a.epilogue != kRowLogits && p.share < kWarps && p.share * 2u <= batches && (p.pairs * p.share * 2u + kWarps - 1u) / kWarps <= most)
        p.share *= 2u;
    const uint32_t grid = std::min<uint32_t>((p.pairs * p.share + kWarps - 1u) / kWarps, most);
    MatvecKernel kernel = a.prologue == kRowPlain
                              ? pick<kRowPlain>(a.epilogue)
                              : (a.prologue == kRowAddNorm
                                     ? pick<kRowAddNorm>(a.epilogue)
                                     : (a.prologue == kRowAddNormNorm ? pick<kRowAddNormNorm>(a.epilogue) : pick<kRowNorm>(a.epilogue)));
    static SmemOptIn once[4][4];
    if (stark_b200_status st = ensure_dynamic_smem(kernel, 200 * 1024, once[a.prologue][a.epilogue])) return st;
    if (a.out_grid) *a.out_grid = grid;
    return launch_chained(kernel, dim3(grid), dim3(kThreads), smem, a.pdl, stream, p);
}

stark_b200_status rows_gemm_f32_launch(const MatrixB16 &w, const float *x, uint32_t m, const float *bias, float *out,
                                       uint32_t ld_out, uint32_t out_cols, cudaStream_t stream, const float *add_scale) {
    if (!w.data || !x || !out || m == 0 || w.cols % 64u != 0) return STARK_B200_INVALID_ARGUMENT;
    rows_gemm_f32_kernel<<<dim3((std::min(w.rows, out_cols) + kTile - 1u) / kTile, (m + kTile - 1u) / kTile), 256, 0, stream>>>(
        w.data, w.rows, w.cols, w.pitch(), x, m, bias, out, ld_out, out_cols, add_scale);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

}  // namespace sb
