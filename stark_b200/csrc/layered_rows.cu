// Row-wise operators of the layered decoders: embedding with a hashed bigram table, the norm of a sublayer's output
// with its residual add, norm of (chosen) rows, gated unit.  One CTA per row; all arithmetic in f32.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kRowThreads = 256;

__global__ void __launch_bounds__(kRowThreads) embed_norm_kernel(EmbedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float row[];
    __shared__ float scratch[32];
    const uint32_t i = blockIdx.x, padded = (a.width + 63u) & ~63u;
    const uint32_t pos = a.tokens ? a.first_pos + i : a.state->position;
    uint32_t token = a.tokens ? a.tokens[i] : a.state->token;
    if (token >= a.vocab) token = 0;  // ids are checked on the host; a greedy pick of a non-finite row is UINT32_MAX
    const uint16_t *src = a.table + (size_t)token * a.ld_table;
    const uint16_t *extra = nullptr;
    if (a.bigram) {
        uint32_t at = a.buckets;  // no previous token
        if (pos != 0u) {
            const uint64_t previous = a.tokens && i != 0u ? a.tokens[i - 1u] : a.history[pos - 1u];
            at = (uint32_t)((previous * a.mul_prev + (uint64_t)token * a.mul_cur) % a.buckets);
        }
        extra = a.bigram + (size_t)at * a.width;
    }
    float s = 0.0f;
    for (uint32_t j = threadIdx.x; j < a.width; j += kRowThreads) {
        float v = bf16_bits_to_f32(src[j]) * a.scale;
        if (extra) v += bf16_bits_to_f32(extra[j]);
        row[j] = v;
        s += v * v;
    }
    const float inv = a.norm_w ? inverse_rms(block_sum(s, scratch), a.width, a.eps) : 1.0f;
    float *x = a.x + (size_t)i * padded;
    for (uint32_t j = threadIdx.x; j < padded; j += kRowThreads) {
        const float v = j < a.width ? row[j] * (a.norm_w ? inv * a.norm_w[j] : 1.0f) : 0.0f;  // its own elements
        x[j] = v;
        if (a.x_b16) a.x_b16[(size_t)i * padded + j] = f32_to_bf16_bits(v);
    }
    if (threadIdx.x == 0) a.history[pos] = token;  // nobody in this launch reads history[first_pos ..]
}

__global__ void __launch_bounds__(kRowThreads) add_norm_rows_kernel(float *x, const float *y, const float *w, uint32_t width,
                                                                    uint32_t padded, float eps, uint16_t *x_b16) {
    extern __shared__ float4 yrow[];
    __shared__ float scratch[32];
    float4 *xr = reinterpret_cast<float4 *>(x + (size_t)blockIdx.x * padded);
    const float4 *yr = reinterpret_cast<const float4 *>(y + (size_t)blockIdx.x * padded);
    const float4 *w4 = reinterpret_cast<const float4 *>(w);
    float s = 0.0f;
    for (uint32_t j = threadIdx.x; j < padded / 4u; j += kRowThreads) {
        const float4 v = yr[j];
        yrow[j] = v;
        s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = inverse_rms(block_sum(s, scratch), width, eps);
    for (uint32_t j = threadIdx.x; j < padded / 4u; j += kRowThreads) {
        const float4 v = yrow[j], g = w4[j];
        float4 o = xr[j];
        o.x += v.x * inv * g.x;
        o.y += v.y * inv * g.y;
        o.z += v.z * inv * g.z;
        o.w += v.w * inv * g.w;
        xr[j] = o;
        if (x_b16)
            reinterpret_cast<uint2 *>(x_b16 + (size_t)blockIdx.x * padded)[j] =
                make_uint2(f32x2_to_bf16x2(o.x, o.y), f32x2_to_bf16x2(o.z, o.w));
    }
}

__global__ void __launch_bounds__(kRowThreads) norm_rows_kernel(const float *x, const uint32_t *rows, const float *w, uint32_t width,
                                                                uint32_t padded, float eps, float *out_f32, uint16_t *out_b16) {
    extern __shared__ float4 xrow[];
    __shared__ float scratch[32];
    const uint32_t i = blockIdx.x;
    const float4 *xr = reinterpret_cast<const float4 *>(x + (size_t)(rows ? rows[i] : i) * padded);
    const float4 *w4 = reinterpret_cast<const float4 *>(w);
    float s = 0.0f;
    for (uint32_t j = threadIdx.x; j < padded / 4u; j += kRowThreads) {
        const float4 v = xr[j];
        xrow[j] = v;
        s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = inverse_rms(block_sum(s, scratch), width, eps);
    for (uint32_t j = threadIdx.x; j < padded / 4u; j += kRowThreads) {
        const float4 v = xrow[j], g = w4[j];
        const float4 o = make_float4(v.x * (inv * g.x), v.y * (inv * g.y), v.z * (inv * g.z), v.w * (inv * g.w));
        if (out_f32) reinterpret_cast<float4 *>(out_f32 + (size_t)i * padded)[j] = o;
        else
            reinterpret_cast<uint2 *>(out_b16 + (size_t)i * padded)[j] = make_uint2(f32x2_to_bf16x2(o.x, o.y), f32x2_to_bf16x2(o.z, o.w));
    }
}

__global__ void __launch_bounds__(256) gate_rows_kernel(const float *gu, uint32_t ld_gu, float *act, uint32_t m, uint32_t ff, Gate gate) {
    const size_t n = (size_t)m * ff;
    for (size_t t = blockIdx.x * 256ull + threadIdx.x; t < n; t += gridDim.x * 256ull) {
        const uint32_t row = (uint32_t)(t / ff), f = (uint32_t)(t % ff);
        const float *src = gu + (size_t)row * ld_gu + (f / 16u) * 32u + f % 16u;
        act[t] = gated(gate, src[0], src[16]);
    }
}

}  // namespace

stark_b200_status embed_norm_launch(const EmbedArgs &a, cudaStream_t stream) {
    if (!a.table || !a.x || !a.history || a.m == 0 || (!a.tokens && (!a.state || a.m != 1u)) ||
        (a.bigram && a.buckets == 0))
        return STARK_B200_INVALID_ARGUMENT;
    const uint32_t smem = pad64(a.width) * 4u;
    static SmemOptIn once;
    if (stark_b200_status st = ensure_dynamic_smem(embed_norm_kernel, 200 * 1024, once)) return st;
    return launch_chained(embed_norm_kernel, dim3(a.m), dim3(kRowThreads), smem, a.pdl, stream, a);
}

stark_b200_status add_norm_rows_launch(float *x, const float *y, const float *w, uint32_t m, uint32_t width, float eps,
                                       uint16_t *x_b16, cudaStream_t stream) {
    static SmemOptIn once;
    if (stark_b200_status st = ensure_dynamic_smem(add_norm_rows_kernel, 200 * 1024, once)) return st;
    add_norm_rows_kernel<<<m, kRowThreads, pad64(width) * 4u, stream>>>(x, y, w, width, pad64(width), eps, x_b16);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

stark_b200_status norm_rows_launch(const float *x, const uint32_t *rows, uint32_t count, const float *w, uint32_t width,
                                   float eps, float *out_f32, uint16_t *out_b16, cudaStream_t stream) {
    static SmemOptIn once;
    if (stark_b200_status st = ensure_dynamic_smem(norm_rows_kernel, 200 * 1024, once)) return st;
    norm_rows_kernel<<<count, kRowThreads, pad64(width) * 4u, stream>>>(x, rows, w, width, pad64(width), eps, out_f32, out_b16);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

stark_b200_status gate_rows_launch(const float *gu, uint32_t ld_gu, float *act, uint32_t m, uint32_t ff_padded, Gate gate,
                                   cudaStream_t stream) {
    const size_t n = (size_t)m * ff_padded;
    gate_rows_kernel<<<(uint32_t)std::min<size_t>((n + 255u) / 256u, 148u * 16u), 256, 0, stream>>>(gu, ld_gu, act, m, ff_padded, gate);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

}  // namespace sb
