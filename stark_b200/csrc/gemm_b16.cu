// Y[M, N] = X[M, K] W[N, K]^T over a bf16 matrix, many rows at a time, on the sm_100a tensor cores (tcgen05.mma,
// accumulators in tensor memory): the prompt-pass contraction of the layered decoders.
//
// The tile shape is that of the 4-bit contraction (prefill_gemm.cu): one CTA owns 256 rows x 256 features (128 rows
// where that leaves SMs idle) and walks K in steps of 64.
//   warp 0      one thread: TMA loads of the step's activation boxes and of the weight box, all bf16 in 128-byte
//               swizzled lines; rows and columns past the ends arrive as zeros
//   warp 1      owns tensor memory; one thread issues the MMAs and commits them to the barrier that frees the stage
//   warps 2-9   the epilogue: bias, then f32 or bf16 rows, or the gate of 16 gate / 16 up columns in turn (columns in front
//               of the gated ones stored as bf16 rows), or a scaled add to f32 rows (the residual stream)
// Every wait is bounded; a wait that runs out sets the error word, the CTA drains and frees its tensor memory.
#include <cuda.h>

#include "layered.cuh"
#include "layered_math.cuh"
#include "tc05.cuh"

namespace sb {

namespace {

constexpr uint32_t kBN = 256, kBK = 64, kStages = 3;
constexpr uint32_t kABox = 128u * 128u;  // 128 rows x 64 bf16
constexpr uint32_t kBStage = kBN * 128u;
constexpr uint32_t kEpilogueWarps = 8, kGemmThreads = (2u + kEpilogueWarps) * 32u;

template <uint32_t HALVES>
struct Tile {
    static constexpr uint32_t kStageBytes = HALVES * kABox + kBStage;
    static constexpr uint32_t kDepth = HALVES == 2u ? kStages : 4u;
    static constexpr uint32_t kSmem = kDepth * kStageBytes + 1024u + 256u;
    static constexpr uint32_t kColumns = HALVES * kBN;
};

// D f32, A and B bf16, both K-major, M 128, N 256
constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((kBN >> 3) << 17) | ((128u >> 4) << 24);

struct GemmB16Params {
    uint32_t steps, m, out_cols, ld_out;
    void *out;
    const float *bias;
    Gate gate;
    uint32_t stored_cols, ld_stored;
    uint16_t *stored_out;
    const float *scale;
    uint32_t *error_word;
};

// 32 f32 values as bf16 into a row, 16-byte aligned.
__device__ inline void store_row32(uint16_t *dst, const uint32_t (&acc)[32]) {
    uint32_t packed[16];
#pragma unroll
    for (int i = 0; i < 32; i += 2) packed[i >> 1] = f32x2_to_bf16x2(__uint_as_float(acc[i]), __uint_as_float(acc[i + 1]));
#pragma unroll
    for (int q = 0; q < 4; ++q)
        reinterpret_cast<uint4 *>(dst)[q] = make_uint4(packed[4 * q], packed[4 * q + 1], packed[4 * q + 2], packed[4 * q + 3]);
}

template <uint32_t HALVES, uint32_t KIND>
__global__ void __launch_bounds__(kGemmThreads, 1)
gemm_b16_kernel(const __grid_constant__ CUtensorMap x_map, const __grid_constant__ CUtensorMap w_map, const GemmB16Params p) {
    using T = Tile<HALVES>;
    extern __shared__ uint8_t gemm_b16_smem[];
    uint8_t *stages = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(gemm_b16_smem) + 1023u) & ~(uintptr_t)1023u);
    uint64_t *bars = reinterpret_cast<uint64_t *>(stages + T::kDepth * T::kStageBytes);
    uint64_t *full = bars, *empty = bars + T::kDepth, *acc_full = bars + 2 * T::kDepth;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(acc_full + 1);
    volatile uint32_t *abort_flag = tmem_slot + 1;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    // row tiles are the fast index: a wave of CTAs then shares few weight tiles, so the weights stream from memory once
    // while the activations of a pass stay in L2
    const uint32_t n0 = blockIdx.y * kBN, m0 = blockIdx.x * (128u * HALVES);

    if (tid == 0) {
        for (uint32_t s = 0; s < T::kDepth; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        mbar_init(acc_full, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(tmem_slot, T::kColumns);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            uint32_t slot = 0, phase = 1;  // a fresh barrier passes a wait on parity 1
            for (uint32_t k = 0; k < p.steps; ++k) {
                if (!mbar_wait_bounded(&empty[slot], phase, abort_flag)) {
                    *abort_flag = 1;
                    atomicOr(p.error_word, kErrMbarTimeout);
                    break;
                }
                uint8_t *stage = stages + slot * T::kStageBytes;
                mbar_arrive_expect_tx(&full[slot], T::kStageBytes);
                tma_load_2d(stage, &x_map, k * kBK, m0, &full[slot]);
                if (HALVES == 2u) tma_load_2d(stage + kABox, &x_map, k * kBK, m0 + 128u, &full[slot]);
                tma_load_2d(stage + HALVES * kABox, &w_map, k * kBK, n0, &full[slot]);
                if (++slot == T::kDepth) slot = 0, phase ^= 1u;
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t slot = 0, phase = 0;
            for (uint32_t k = 0; k < p.steps; ++k) {
                if (!mbar_wait_bounded(&full[slot], phase, abort_flag)) {
                    *abort_flag = 1;
                    atomicOr(p.error_word, kErrMbarTimeout);
                    break;
                }
                tc_fence_after();
                const uint32_t a_addr = smem_u32(stages + slot * T::kStageBytes), b_addr = a_addr + HALVES * kABox;
#pragma unroll
                for (uint32_t half = 0; half < HALVES; ++half)
#pragma unroll
                    for (uint32_t k4 = 0; k4 < kBK / 16u; ++k4)
                        umma_f16(tmem_base + half * kBN, smem_desc_sw128(a_addr + half * kABox + k4 * 32u),
                                 smem_desc_sw128(b_addr + k4 * 32u), kIdesc, (k | k4) != 0u ? 1u : 0u);
                umma_commit(&empty[slot]);
                if (++slot == T::kDepth) slot = 0, phase ^= 1u;
            }
            umma_commit(acc_full);  // also on the give-up path: the epilogue warps wait on it
        }
    } else {
        // warp -> (sub-partition, accumulator half); with one accumulator two warps share a sub-partition's columns
        const uint32_t d = warp - 2u, sub = warp & 3u, half = HALVES == 2u ? d >> 2 : 0u;
        const uint32_t c_first = HALVES == 2u ? 0u : (d >> 2) * (kBN / 64u), c_count = kBN / 32u / (3u - HALVES);
        const bool acc_ok = mbar_wait_bounded(acc_full, 0, abort_flag);
        if (!acc_ok && lane == 0) atomicOr(p.error_word, kErrMbarTimeout);
        tc_fence_after();
        const uint32_t row = m0 + half * 128u + sub * 32u + lane;
        const bool row_ok = row < p.m && acc_ok;
#pragma unroll 1
        for (uint32_t c = c_first; c < c_first + c_count; ++c) {
            const uint32_t f0 = n0 + c * 32u;
            if (f0 >= p.out_cols) break;
            uint32_t acc[32];
            tmem_ld_32x32(tmem_base + ((sub * 32u) << 16) + half * kBN + c * 32u, acc);
            const bool whole = f0 + 32u <= p.out_cols;
            if (p.bias) {  // biases come with gated and stored layers whose widths are whole blocks
#pragma unroll
                for (int i = 0; i < 32; i += 4) {
                    const float4 b = __ldg(reinterpret_cast<const float4 *>(p.bias + f0 + i));
                    acc[i] = __float_as_uint(__uint_as_float(acc[i]) + b.x);
                    acc[i + 1] = __float_as_uint(__uint_as_float(acc[i + 1]) + b.y);
                    acc[i + 2] = __float_as_uint(__uint_as_float(acc[i + 2]) + b.z);
                    acc[i + 3] = __float_as_uint(__uint_as_float(acc[i + 3]) + b.w);
                }
            }
            if (!row_ok) continue;
            if (KIND == kGemmGate) {
                if (f0 < p.stored_cols) {
                    store_row32(p.stored_out + (size_t)row * p.ld_stored + f0, acc);
                    continue;
                }
                uint32_t packed[8];
#pragma unroll
                for (int i = 0; i < 16; i += 2)
                    packed[i >> 1] = f32x2_to_bf16x2(gated(p.gate, __uint_as_float(acc[i]), __uint_as_float(acc[16 + i])),
                                                     gated(p.gate, __uint_as_float(acc[i + 1]), __uint_as_float(acc[17 + i])));
                uint4 *dst = reinterpret_cast<uint4 *>(static_cast<uint16_t *>(p.out) + (size_t)row * p.ld_out + (f0 - p.stored_cols) / 2u);
                dst[0] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
                dst[1] = make_uint4(packed[4], packed[5], packed[6], packed[7]);
            } else if (KIND == kGemmBf16) {
                store_row32(static_cast<uint16_t *>(p.out) + (size_t)row * p.ld_out + f0, acc);
            } else if (KIND == kGemmResidual) {
                float4 *dst = reinterpret_cast<float4 *>(static_cast<float *>(p.out) + (size_t)row * p.ld_out + f0);
                const float4 *scale = reinterpret_cast<const float4 *>(p.scale + f0);
                float4 v[8];
#pragma unroll
                for (int q = 0; q < 8; ++q) v[q] = dst[q];
#pragma unroll
                for (int q = 0; q < 8; ++q) {
                    const float4 g = __ldg(scale + q);
                    v[q].x = fmaf(g.x, __uint_as_float(acc[4 * q]), v[q].x);
                    v[q].y = fmaf(g.y, __uint_as_float(acc[4 * q + 1]), v[q].y);
                    v[q].z = fmaf(g.z, __uint_as_float(acc[4 * q + 2]), v[q].z);
                    v[q].w = fmaf(g.w, __uint_as_float(acc[4 * q + 3]), v[q].w);
                    dst[q] = v[q];
                }
            } else {
                float *dst = static_cast<float *>(p.out) + (size_t)row * p.ld_out + f0;
                if (whole && p.ld_out % 4u == 0) {
#pragma unroll
                    for (int q = 0; q < 8; ++q)
                        reinterpret_cast<uint4 *>(dst)[q] = make_uint4(acc[4 * q], acc[4 * q + 1], acc[4 * q + 2], acc[4 * q + 3]);
                } else {
#pragma unroll
                    for (uint32_t i = 0; i < 32u; ++i)
                        if (f0 + i < p.out_cols) dst[i] = __uint_as_float(acc[i]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, T::kColumns);
    }
}

using GemmB16Kernel = void (*)(const CUtensorMap, const CUtensorMap, const GemmB16Params);
template <uint32_t HALVES>
stark_b200_status launch(const GemmB16Args &a, const CUtensorMap &x_map, const CUtensorMap &w_map, const GemmB16Params &p,
                         cudaStream_t stream) {
    using T = Tile<HALVES>;
    auto kernel = a.kind == kGemmBf16
                      ? gemm_b16_kernel<HALVES, kGemmBf16>
                      : (a.kind == kGemmF32 ? gemm_b16_kernel<HALVES, kGemmF32>
                                            : (a.kind == kGemmGate ? gemm_b16_kernel<HALVES, kGemmGate> : gemm_b16_kernel<HALVES, kGemmResidual>));
    static SmemOptIn once[4];
    if (stark_b200_status st = ensure_dynamic_smem(kernel, (int)T::kSmem, once[a.kind])) return st;
    kernel<<<dim3((a.m + 128u * HALVES - 1u) / (128u * HALVES), (a.out_cols + kBN - 1u) / kBN), kGemmThreads, T::kSmem, stream>>>(
        x_map, w_map, p);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

}  // namespace

stark_b200_status gemm_b16_launch(const GemmB16Args &a, cudaStream_t stream) {
    if (!a.w.data || !a.x || !a.out || a.m == 0 || a.m > a.x_rows || a.w.cols % kBK || a.ld_x % 8u || a.ld_x < a.w.cols ||
        a.out_cols > a.w.rows || (reinterpret_cast<uintptr_t>(a.x) & 15u))
        return STARK_B200_INVALID_ARGUMENT;
    // vector stores and bias reads work on whole 32-column blocks; only a bare f32 output may end inside one
    if ((a.kind != kGemmF32 || a.bias) && (a.out_cols % 32u || a.ld_out % 16u)) return STARK_B200_INVALID_ARGUMENT;
    if (a.kind == kGemmGate && a.stored_cols && (!a.stored_out || a.stored_cols % 32u || a.ld_stored % 16u)) return STARK_B200_INVALID_ARGUMENT;
    if (a.kind == kGemmResidual && (!a.scale || a.bias)) return STARK_B200_INVALID_ARGUMENT;
    DeviceContext *ctx = device_context();
    EncodeTiledFn encode = encode_tiled();
    if (!ctx || !encode) return STARK_B200_DEVICE_FAILURE;
    const cuuint32_t elem[2] = {1u, 1u};
    CUtensorMap x_map, w_map;
    auto make = [&](CUtensorMap *map, const uint16_t *base, uint32_t rows, uint32_t ld, uint32_t box_rows) {
        const cuuint64_t dims[2] = {a.w.cols, rows}, strides[1] = {(cuuint64_t)ld * 2u};
        const cuuint32_t box[2] = {kBK, box_rows};
        return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<uint16_t *>(base), dims, strides, box, elem,
                      CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                      CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
    };
    if (!make(&x_map, a.x, a.x_rows, a.ld_x, 128u) || !make(&w_map, a.w.data, a.w.rows, a.w.pitch(), kBN))
        return STARK_B200_DEVICE_FAILURE;
    const GemmB16Params p{a.w.cols / kBK, a.m, a.out_cols, a.ld_out, a.out, a.bias, a.gate, a.kind == kGemmGate ? a.stored_cols : 0u,
                          a.ld_stored, a.stored_out, a.scale, ctx->error_word};
    // 256-row tiles unless 128-row tiles fill the SMs so much better that it pays for their loading the weight tile
    // once per 128 rows (a fifth slower per row)
    const uint32_t wide = (a.out_cols + kBN - 1u) / kBN, tall = (a.m + 255u) / 256u, flat = (a.m + 127u) / 128u;
    const uint32_t waves2 = (wide * tall + 147u) / 148u * 2u, waves1 = (wide * flat + 147u) / 148u;
    return waves1 * 5u < waves2 * 4u ? launch<1>(a, x_map, w_map, p, stream) : launch<2>(a, x_map, w_map, p, stream);
}

}  // namespace sb
