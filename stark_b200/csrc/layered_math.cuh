// Device arithmetic and the launch helper shared by the layered decoders' kernels.
#pragma once
#include <algorithm>
#include <cmath>

#include "common.cuh"

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
