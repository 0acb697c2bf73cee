// Latent attention in its absorbed form: the cache holds one row per position -- the normed latent c and a rotated key
// part all heads share -- and the per-head key and value matrices are applied on the query's and the output's side:
//   score_j = ((W_uk^T q) . c_j + q_rot . r_j) * scale,     out = W_uv (sum_j a_j c_j)
// so a decode step reads rank + rot values per cached row whatever the number of heads.  Three launches:
//   latent_query    per head and 64 latent columns: W_uk^T q, the rotated query part, both times scale * log2(e); one
//                   more CTA per row norms the new latent, rotates the new key part and appends the cache row
//   latent_attend   per span of the cached rows and group of heads: f32 scores, running softmax, weighted latents
//   latent_value    per head and 64 output values: merge of the spans, then W_uv
// Angles, norms, scores and softmax are f32.  A row of a pass attends to the rows up to its own position.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kQueryThreads = 256;
__device__ inline float *partial_of(const LatentArgs &a, uint32_t row, uint32_t head, uint32_t split) {
    return a.partials + (((size_t)row * a.s.heads + head) * a.splits + split) * (a.s.rank_p + 4u);
}

// The new cache row of one position: latent / rms * w, and the key part rotated.  One CTA.
template <typename T, typename C>
__device__ void append_row(const LatentArgs &a, const T *src, uint32_t pos, float *scratch) {
    const LatentShape &s = a.s;
    C *dst = reinterpret_cast<C *>(a.cache) +
             ((size_t)a.block_table[pos / kPageTokens] * kPageTokens + pos % kPageTokens) * s.row();
    float sum = 0.0f;
    for (uint32_t i = threadIdx.x; i < s.rank; i += blockDim.x) {
        const float v = load_value(src + i);
        sum += v * v;
    }
    const float inv = inverse_rms(block_sum(sum, scratch), s.rank, a.eps);
    for (uint32_t i = threadIdx.x; i < s.rank_p; i += blockDim.x)
        store_value(dst + i, i < s.rank ? load_value(src + i) * inv * a.latent_norm[i] : 0.0f);
    for (uint32_t i = threadIdx.x; i < s.rot_p / 2u; i += blockDim.x) {
        float u = load_value(src + s.rank_p + 2u * i), v = load_value(src + s.rank_p + 2u * i + 1u);
        if (i < a.rot.pairs) {
            float sn, cs;
            sincosf((float)pos * a.rot.freq[i], &sn, &cs);
            sn *= a.rot.factor, cs *= a.rot.factor;
            const float u0 = u;
            u = u0 * cs - v * sn;
            v = v * cs + u0 * sn;
        }
        store_value(dst + s.rank_p + 2u * i, u);
        store_value(dst + s.rank_p + 2u * i + 1u, v);
    }
}

// blockIdx.x: (head, 64 latent columns), then one CTA that appends the cache row; blockIdx.y: row
template <typename T, typename C>
__global__ void __launch_bounds__(kQueryThreads) latent_query_kernel(const LatentArgs a) {
    extern __shared__ float q[];                 // [dim_p]
    __shared__ float part[32][64];
    __shared__ float scratch[32];
    const LatentShape &s = a.s;
    const uint32_t blocks = s.rank_p / 64u, head = blockIdx.x / blocks, piece = blockIdx.x % blocks;
    const uint32_t row = blockIdx.y, lane8 = threadIdx.x & 7u, slice = threadIdx.x >> 3;
    // this thread's first weights do not depend on the previous kernel
    const uint16_t *uk = a.uk_uv.data + (size_t)head * s.dim_p * s.rank_p + piece * 64u + lane8 * 8u;
    uint4 w[4];
    if (head < s.heads) {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j) {
            const uint32_t d = slice + 32u * j;
            w[j] = d < s.dim_p ? ldg_nc_v4(uk + (size_t)d * s.rank_p) : make_uint4(0u, 0u, 0u, 0u);
        }
    }
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t pos = a.state ? a.state->position : a.first_pos + row;
    const T *src = reinterpret_cast<const T *>(a.qd) + (size_t)row * a.ld_qd;
    if (head >= s.heads) {
        append_row<T, C>(a, src + s.q_width(), pos, scratch);
        return;
    }
    const float factor = a.scale * kLog2e;
    float *dst = a.queries + ((size_t)row * s.heads + head) * s.row();
    const T *qh = src + (size_t)head * s.q_head();
    for (uint32_t i = threadIdx.x; i < s.dim_p; i += kQueryThreads) q[i] = load_value(qh + i);
    if (piece == 0u) {
        for (uint32_t i = threadIdx.x; i < s.rot_p / 2u; i += kQueryThreads) {
            float u = load_value(qh + s.dim_p + 2u * i), v = load_value(qh + s.dim_p + 2u * i + 1u);
            if (i < a.rot.pairs) {
                float sn, cs;
                sincosf((float)pos * a.rot.freq[i], &sn, &cs);
                sn *= a.rot.factor, cs *= a.rot.factor;
                const float u0 = u;
                u = u0 * cs - v * sn;
                v = v * cs + u0 * sn;
            }
            dst[s.rank_p + 2u * i] = u * factor;
            dst[s.rank_p + 2u * i + 1u] = v * factor;
        }
    }
    __syncthreads();
    float acc[8] = {};
    for (uint32_t d0 = 0; d0 < s.dim_p; d0 += 128u) {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j) {
            const uint32_t d = d0 + slice + 32u * j;
            if (d >= s.dim_p) break;
            const uint4 v = d0 == 0u ? w[j] : ldg_nc_v4(uk + (size_t)d * s.rank_p);
            const uint32_t words[4] = {v.x, v.y, v.z, v.w};
            const float x = q[d];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                acc[2 * e] = fmaf(__uint_as_float(words[e] << 16), x, acc[2 * e]);
                acc[2 * e + 1] = fmaf(__uint_as_float(words[e] & 0xffff0000u), x, acc[2 * e + 1]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) part[slice][lane8 * 8u + e] = acc[e];
    __syncthreads();
    if (threadIdx.x < 64u) {
        float sum = 0.0f;
#pragma unroll
        for (uint32_t k = 0; k < 32u; ++k) sum += part[k][threadIdx.x];
        dst[piece * 64u + threadIdx.x] = sum * factor;
    }
}

// blockIdx.x: (head, 64 output values), blockIdx.y: row
template <typename O>
__global__ void __launch_bounds__(256) latent_value_kernel(const LatentArgs a) {
    extern __shared__ __align__(16) float o[];  // [rank_p], then the pieces of the merge
    __shared__ float weight[kMaxSplits];
    const LatentShape &s = a.s;
    const uint32_t blocks = s.vdim_p / 64u, head = blockIdx.x / blocks, piece = blockIdx.x % blocks, row = blockIdx.y;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    const uint16_t *uv = a.uk_uv.data + ((size_t)s.heads * s.dim_p + (size_t)head * s.vdim_p + piece * 64u + warp * 8u) * s.rank_p;
    // the first 256 columns of this warp's eight rows: weights do not depend on the previous kernel
    uint4 w[8];
#pragma unroll
    for (uint32_t j = 0; j < 8u; ++j)
        w[j] = lane * 8u < s.rank_p ? ldg_nc_v4(uv + (size_t)j * s.rank_p + lane * 8u) : make_uint4(0u, 0u, 0u, 0u);
    pdl_launch_dependents();
    pdl_wait();
    const float *part = partial_of(a, row, head, 0);
    const uint32_t pitch = s.rank_p + 4u;
    // every warp forms the spans' weights exp2(m - max) / sum for itself; the first one leaves them for the columns
    {
        float m[2], l[2], top = -INFINITY, sum = 0.0f;
#pragma unroll
        for (uint32_t j = 0; j < 2u; ++j) {
            const uint32_t k = lane + 32u * j;
            const float2 v = k < a.splits ? *reinterpret_cast<const float2 *>(part + (size_t)k * pitch) : make_float2(-INFINITY, 0.0f);
            m[j] = v.x, l[j] = v.y;
            top = fmaxf(top, v.x);
        }
        top = warp_max(top);
#pragma unroll
        for (uint32_t j = 0; j < 2u; ++j) {
            m[j] = exp2f(m[j] - top);  // 0 for an empty span
            sum = fmaf(m[j], l[j], sum);
        }
        const float inv = 1.0f / warp_sum(sum);
        if (warp == 0u) weight[lane] = m[0] * inv, weight[lane + 32u] = m[1] * inv;
    }
    __syncthreads();
    // four columns a thread; where the latent is narrow several threads share the spans of the same four
    const uint32_t quads = s.rank_p / 4u, shares = quads >= 256u ? 1u : 256u / quads;
    float4 *pieces = reinterpret_cast<float4 *>(o + s.rank_p);  // [shares][quads]
    for (uint32_t t = threadIdx.x; t < quads * shares; t += 256u) {
        const uint32_t quad = t % quads, share = t / quads;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
        for (uint32_t k = share; k < a.splits; k += shares) {
            const float4 x = *reinterpret_cast<const float4 *>(part + (size_t)k * pitch + 4u + quad * 4u);
            const float c = weight[k];
            v.x = fmaf(c, x.x, v.x), v.y = fmaf(c, x.y, v.y), v.z = fmaf(c, x.z, v.z), v.w = fmaf(c, x.w, v.w);
        }
        pieces[t] = v;
    }
    __syncthreads();
    for (uint32_t quad = threadIdx.x; quad < quads; quad += 256u) {
        float4 v = pieces[quad];
        for (uint32_t k = 1; k < shares; ++k) {
            const float4 x = pieces[k * quads + quad];
            v.x += x.x, v.y += x.y, v.z += x.z, v.w += x.w;
        }
        reinterpret_cast<float4 *>(o)[quad] = v;
    }
    __syncthreads();
    float acc[8] = {};
    for (uint32_t c = lane * 8u; c < s.rank_p; c += 256u) {
        const float4 x = *reinterpret_cast<const float4 *>(o + c), y = *reinterpret_cast<const float4 *>(o + c + 4u);
#pragma unroll
        for (uint32_t j = 0; j < 8u; ++j) {
            const uint4 v = c < 256u ? w[j] : ldg_nc_v4(uv + (size_t)j * s.rank_p + c);
            acc[j] = fmaf(__uint_as_float(v.x << 16), x.x, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.x & 0xffff0000u), x.y, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.y << 16), x.z, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.y & 0xffff0000u), x.w, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.z << 16), y.x, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.z & 0xffff0000u), y.y, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.w << 16), y.z, acc[j]);
            acc[j] = fmaf(__uint_as_float(v.w & 0xffff0000u), y.w, acc[j]);
        }
    }
    O *dst = reinterpret_cast<O *>(a.out) + ((size_t)row * s.heads + head) * s.vdim_p + piece * 64u + warp * 8u;
#pragma unroll
    for (uint32_t j = 0; j < 8u; ++j) {
        const float v = warp_sum(acc[j]);
        if (lane == 0) store_value(dst + j, v);
    }
}

// One CTA per row of a pass: the new cache row, and the rotated part of every query head rotated in place (bf16 rows).
__global__ void __launch_bounds__(256) latent_rotate_append_kernel(const LatentArgs a) {
    extern __shared__ float2 turn[];  // [pairs] (cos, sin)
    __shared__ float scratch[32];
    const LatentShape &s = a.s;
    const uint32_t row = blockIdx.x, pos = a.first_pos + row;
    uint16_t *src = const_cast<uint16_t *>(reinterpret_cast<const uint16_t *>(a.qd)) + (size_t)row * a.ld_qd;
    for (uint32_t i = threadIdx.x; i < a.rot.pairs; i += 256u) {
        float sn, cs;
        sincosf((float)pos * a.rot.freq[i], &sn, &cs);
        turn[i] = make_float2(cs * a.rot.factor, sn * a.rot.factor);
    }
    append_row<uint16_t, uint16_t>(a, src + s.q_width(), pos, scratch);
    __syncthreads();
    for (uint32_t t = threadIdx.x; t < s.heads * a.rot.pairs; t += 256u) {
        const uint32_t head = t / a.rot.pairs, i = t % a.rot.pairs;
        uint32_t *pair = reinterpret_cast<uint32_t *>(src + (size_t)head * s.q_head() + s.dim_p) + i;
        const float u = __uint_as_float(*pair << 16), v = __uint_as_float(*pair & 0xffff0000u);
        *pair = f32x2_to_bf16x2(u * turn[i].x - v * turn[i].y, v * turn[i].x + u * turn[i].y);
    }
}

stark_b200_status check_args(const LatentArgs &a) {
    if (!latent_shape_supported(a.s)) return STARK_B200_UNSUPPORTED;
    if (!a.qd || !a.cache || !a.block_table || !a.uk_uv.data || a.m == 0 || (a.state && a.m != 1u) || !a.rot.freq ||
        a.splits > kMaxSplits || a.splits == 0)
        return STARK_B200_INVALID_ARGUMENT;
    return STARK_B200_OK;
}

}  // namespace

bool latent_shape_supported(const LatentShape &s) {
    return s.heads != 0 && s.dim != 0 && s.rot_dim % 2u == 0 && s.vdim != 0 && s.rank != 0 &&
           span_attend_supports(s.row(), s.rank_p) && s.dim_p <= 4096u;
}

stark_b200_status latent_query_launch(const LatentArgs &a, cudaStream_t stream) {
    if (stark_b200_status st = check_args(a)) return st;
    if (!a.queries) return STARK_B200_INVALID_ARGUMENT;
    const dim3 grid(a.s.heads * (a.s.rank_p / 64u) + 1u, a.m);
    auto kernel = a.qd_b16 ? (a.cache_f32 ? latent_query_kernel<uint16_t, float> : latent_query_kernel<uint16_t, uint16_t>)
                           : (a.cache_f32 ? latent_query_kernel<float, float> : latent_query_kernel<float, uint16_t>);
    return launch_chained(kernel, grid, dim3(kQueryThreads), a.s.dim_p * 4u, a.pdl, stream, a);
}

stark_b200_status latent_attend_launch(const LatentArgs &a, cudaStream_t stream) {
    if (stark_b200_status st = check_args(a)) return st;
    if (!a.queries || !a.partials) return STARK_B200_INVALID_ARGUMENT;
    if (!a.cache_f32 && latent_attend_mma_supports(a.s)) return latent_attend_mma_launch(a, stream);
    if (a.cluster != 1u) return STARK_B200_INVALID_ARGUMENT;
    SpanAttendArgs g{};  // all heads share the cached rows; their values are the latent columns of the same rows
    g.queries = a.queries, g.heads = a.s.heads, g.key_heads = 1, g.width = a.s.row(), g.out_width = a.s.rank_p;
    g.keys = g.values = a.cache, g.key_pitch = g.value_pitch = a.s.row(), g.cache_f32 = a.cache_f32;
    g.block_table = a.block_table, g.state = a.state, g.first_pos = a.first_pos, g.m = a.m, g.splits = a.splits;
    g.partials = a.partials, g.pdl = a.pdl;
    return span_attend_launch(g, stream);
}

stark_b200_status latent_value_launch(const LatentArgs &a, cudaStream_t stream) {
    if (stark_b200_status st = check_args(a)) return st;
    if (!a.partials || !a.out) return STARK_B200_INVALID_ARGUMENT;
    auto kernel = a.out_b16 ? latent_value_kernel<uint16_t> : latent_value_kernel<float>;
    return launch_chained(kernel, dim3(a.s.heads * (a.s.vdim_p / 64u), a.m), dim3(256),
                          a.s.rank_p * 4u + std::max(a.s.rank_p * 4u, 4096u), a.pdl, stream, a);
}

stark_b200_status latent_rotate_append_launch(const LatentArgs &a, cudaStream_t stream) {
    if (stark_b200_status st = check_args(a)) return st;
    if (a.cache_f32 || !a.qd_b16) return STARK_B200_INVALID_ARGUMENT;
    latent_rotate_append_kernel<<<a.m, 256, a.s.rot_p * 4u, stream>>>(a);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

}  // namespace sb
