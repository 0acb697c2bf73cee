// Device arithmetic and the launch helper shared by the layered decoders' kernels.
#pragma once
#include <algorithm>
#include <cmath>

#include "layered.cuh"

namespace sb {

// Sum over the CTA's threads, the same value in every thread (whole warps, at most 32 of them).
__device__ inline float block_sum(float v, float *scratch /* [32] */) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31u) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float r = 0.0f;
    for (uint32_t w = 0; w < blockDim.x / 32u; ++w) r += scratch[w];
    return r;
}

__device__ inline float inverse_rms(float sum_of_squares, uint32_t width, float eps) {
    return 1.0f / sqrtf(sum_of_squares / (float)width + eps);
}

// Gated unit with clamped halves and a shifted up half: g = min(g, limit), u = clamp(u, -limit, limit),
// g * sigmoid(1.702 g) * (u + 1).
__device__ inline float clamped_gate(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}

__device__ inline float gated(const Gate &gate, float g, float u) {
    return gate.kind == kGateSilu ? g / (1.0f + expf(-g)) * u : clamped_gate(g, u, gate.limit);
}

constexpr float kLog2e = 1.4426950408889634f;

template <typename T>
__device__ inline float load_value(const T *p);
template <>
__device__ inline float load_value<float>(const float *p) { return *p; }
template <>
__device__ inline float load_value<uint16_t>(const uint16_t *p) { return bf16_bits_to_f32(*p); }
__device__ inline void store_value(float *p, float v) { *p = v; }
__device__ inline void store_value(uint16_t *p, float v) { *p = f32_to_bf16_bits(v); }
// Two neighbours at an even index.
__device__ inline float2 load_pair(const float *p) { return *reinterpret_cast<const float2 *>(p); }
__device__ inline float2 load_pair(const uint16_t *p) {
    const uint32_t w = *reinterpret_cast<const uint32_t *>(p);
    return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u));
}
__device__ inline void store_pair(float *p, float2 v) { *reinterpret_cast<float2 *>(p) = v; }
__device__ inline void store_pair(uint16_t *p, float2 v) { *reinterpret_cast<uint32_t *>(p) = f32x2_to_bf16x2(v.x, v.y); }

// The values the first mixing layer leaves for the later ones: a row without padding, [groups * vdim], so that layers that
// divide it into other heads mix the same entries.  `o` holds entries c and c + 1 of a head of n, c even.
__device__ inline void keep_first_values(float *head, uint32_t c, uint32_t n, float2 o) {
    if (c < n) head[c] = o.x;
    if (c + 1u < n) head[c + 1u] = o.y;
}
__device__ inline float2 mix_values(const float *head, uint32_t c, uint32_t n, float2 o, float share) {
    if (c < n) o.x = (1.0f - share) * o.x + share * head[c];
    if (c + 1u < n) o.y = (1.0f - share) * o.y + share * head[c + 1u];
    return o;
}

// Factor on the queries of a position: 1 + coef * ln((position + 1) / every + 1), whole division.
__host__ __device__ inline float query_temperature(uint32_t position, float coef, uint32_t every) {
    return 1.0f + coef * logf((float)((position + 1u) / every + 1u));
}

template <typename... Params, typename... Args>
inline stark_b200_status launch_chained(void (*kernel)(Params...), dim3 grid, dim3 block, uint32_t smem, bool pdl,
                                        cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 1 : 0;
    SB_CUDA(cudaLaunchKernelEx(&cfg, kernel, static_cast<Params>(args)...));
    return STARK_B200_OK;
}

}  // namespace sb
