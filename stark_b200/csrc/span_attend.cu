// Attention of one or a few rows over spans of a paged cache on the CUDA cores, and the merge of the spans: f32 scores and
// softmax over an f32 or bf16 cache, any head sizes.  The tensor-core forms beside it serve bf16 caches of common sizes.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kThreads = 256, kColumns = 8;  // value columns per thread: up to 2048

__device__ inline float *partial_of(const SpanAttendArgs &a, uint32_t row, uint32_t head, uint32_t split) {
    return a.partials + (((size_t)row * a.heads + head) * a.splits + split) * (a.out_width + 4u);
}

// One head of one row over one span of whole pages.  blockIdx: (span, head, row)
template <typename C>
__global__ void __launch_bounds__(kThreads) span_attend_kernel(const SpanAttendArgs a) {
    extern __shared__ float q[];  // [width]
    __shared__ float p[kPageTokens];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t split = blockIdx.x, head = blockIdx.y, row = blockIdx.z, width = a.width;
    const uint32_t key_head = head / (a.heads / a.key_heads);
    const uint32_t pos = a.state ? a.state->position : a.first_pos + row;
    const uint32_t pages = pos / kPageTokens + 1u, span = (pages + a.splits - 1u) / a.splits;
    const uint32_t lo = min(pages, split * span), hi = min(pages, lo + span);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    const float *src = a.queries + ((size_t)row * a.heads + head) * width;
    for (uint32_t i = threadIdx.x; i < width; i += kThreads) q[i] = src[i];
    float m = -INFINITY, l = 0.0f, acc[kColumns] = {};
    for (uint32_t page = lo; page < hi; ++page) {
        const size_t first = ((size_t)a.block_table[page] * a.key_heads + key_head) * kPageTokens;
        const C *keys = reinterpret_cast<const C *>(a.keys) + first * a.key_pitch;
        const C *values = reinterpret_cast<const C *>(a.values) + first * a.value_pitch;
        __syncthreads();
        for (uint32_t k = warp; k < kPageTokens; k += kThreads / 32u) {
            float dot = -INFINITY;
            if (page * kPageTokens + k <= pos) {
                dot = 0.0f;
                for (uint32_t i = lane; i < width; i += 32u) dot = fmaf(q[i], load_value(keys + (size_t)k * a.key_pitch + i), dot);
                dot = warp_sum(dot);
            }
            if (lane == 0) p[k] = dot;
        }
        __syncthreads();
        float top = m;
        for (uint32_t k = 0; k < kPageTokens; ++k) top = fmaxf(top, p[k]);
        const float keep = exp2f(m - top);  // 0 on the first page
        m = top;
        l *= keep;
#pragma unroll
        for (uint32_t c = 0; c < kColumns; ++c) acc[c] *= keep;
        for (uint32_t k = 0; k < kPageTokens; ++k) {
            if (page * kPageTokens + k > pos) break;
            const float w = exp2f(p[k] - top);
            l += w;
#pragma unroll
            for (uint32_t c = 0; c < kColumns; ++c) {
                const uint32_t i = threadIdx.x + c * kThreads;
                if (i < a.out_width) acc[c] = fmaf(w, load_value(values + (size_t)k * a.value_pitch + i), acc[c]);
            }
        }
    }
    float *dst = partial_of(a, row, head, split);
    if (threadIdx.x == 0) dst[0] = m, dst[1] = l;
#pragma unroll
    for (uint32_t c = 0; c < kColumns; ++c) {
        const uint32_t i = threadIdx.x + c * kThreads;
        if (i < a.out_width) dst[4u + i] = acc[c];
    }
}

// blockIdx: (head, row)
template <typename O>
__global__ void __launch_bounds__(128) span_merge_kernel(const SpanAttendArgs a) {
    __shared__ float weight[kMaxSplits];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t head = blockIdx.x, row = blockIdx.y, lane = threadIdx.x & 31u, pitch = a.out_width + 4u;
    const float *part = partial_of(a, row, head, 0);
    if (threadIdx.x < 32u) {
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
        weight[lane] = m[0] * inv, weight[lane + 32u] = m[1] * inv;
    }
    __syncthreads();
    O *dst = reinterpret_cast<O *>(a.out) + (size_t)row * a.ld_out + (size_t)head * a.out_width;
    for (uint32_t i = threadIdx.x; i < a.out_width; i += 128u) {
        float v = 0.0f;
        for (uint32_t k = 0; k < a.splits; ++k) v = fmaf(weight[k], part[(size_t)k * pitch + 4u + i], v);
        store_value(dst + i, v);
    }
}

bool valid(const SpanAttendArgs &a) {
    return span_attend_supports(a.width, a.out_width) && a.heads && a.key_heads && a.heads % a.key_heads == 0 && a.m &&
           a.splits && a.splits <= kMaxSplits && a.partials && !(a.state && a.m != 1u);
}

}  // namespace

bool span_attend_supports(uint32_t width, uint32_t out_width) {
    return width && width <= 4096u && out_width && out_width % 4u == 0 && out_width <= kThreads * kColumns;
}

stark_b200_status span_attend_launch(const SpanAttendArgs &a, cudaStream_t stream) {
    if (!valid(a) || !a.queries || !a.keys || !a.values || !a.block_table) return STARK_B200_INVALID_ARGUMENT;
    auto kernel = a.cache_f32 ? span_attend_kernel<float> : span_attend_kernel<uint16_t>;
    return launch_chained(kernel, dim3(a.splits, a.heads, a.m), dim3(kThreads), a.width * 4u, a.pdl, stream, a);
}

stark_b200_status span_merge_launch(const SpanAttendArgs &a, cudaStream_t stream) {
    if (!valid(a) || !a.out) return STARK_B200_INVALID_ARGUMENT;
    auto kernel = a.out_b16 ? span_merge_kernel<uint16_t> : span_merge_kernel<float>;
    return launch_chained(kernel, dim3(a.heads, a.m), dim3(128), 0, a.pdl, stream, a);
}

}  // namespace sb
