// Causal attention of a prompt pass on the sm_100a tensor cores (tcgen05.mma, accumulators in tensor memory) for the layered
// decoders' mixers.
//
// The scheme is that of prefill_attention_tc.cu -- one CTA owns 128 rows of one head and walks the keys twice, first for
// every row's maximum, then P = exp2(S - max) and O += P V with P as bf16 hi + lo, so no accumulator is ever rescaled --
// with three things of its own: query and value widths are arguments (whole blocks of 64, up to 256); the key tile of a
// step may be put together from two places (blocks of the head's own, blocks every head shares); and where the scores are
// bounded beforehand (queries and keys of unit root mean square) the bound stands in for the maximum and the keys are
// walked once.  A step is one cache page (64 keys), which leaves room for three key stages at 192-wide queries.
// Latent attention comes in the expanded form: keys W_uk c and values W_uv c of every visible row were formed by one
// contraction over the cache, the rotated key part comes from the cache itself.  Grouped-query attention reads its pages.
//   warps 0-7   softmax: thread = row (tensor-memory lane) x half of the step's keys
//   warp 8      one thread: TMA loads
//   warp 9      owns tensor memory; one thread issues the MMAs
// Every wait is bounded; a wait that runs out sets the error word, the CTA drains and frees its tensor memory.
#include <cuda.h>

#include <algorithm>

#include "device_math.cuh"
#include "layered.cuh"
#include "layered_math.cuh"
#include "tc05.cuh"

namespace sb {

namespace {

constexpr uint32_t kKeys = kPageTokens;       // keys per step
constexpr uint32_t kKeyBlock = kKeys * 128u;  // 64 keys x 64 elements: 8 KB
constexpr uint32_t kRowBlock = 128u * 128u;   // 128 rows x 64 elements: 16 KB
constexpr uint32_t kSoftmaxWarps = 8, kThreads = (kSoftmaxWarps + 2u) * 32u;
constexpr uint32_t kMaxKeyStages = 3, kValueStages = 2;
constexpr uint32_t kMaxBlocks = 4;            // widths up to 256
constexpr uint32_t kTail = 2048u;             // barriers, exchange words
constexpr uint32_t kTmemColumns = 512, kOutColumn = 128;  // S twice (2 x 64), O from column 128 (up to 256)
constexpr uint32_t kIdescBase = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24);
constexpr uint32_t kIdescS = kIdescBase | ((kKeys >> 3) << 17);
constexpr uint32_t kIdescPV = kIdescBase | (1u << 16);  // B (the values) MN-major; N is added at run time

__device__ inline float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct AttendTcParams {
    uint16_t *out;
    const int32_t *block_table;
    uint32_t m, first_pos, heads, key_heads;
    uint32_t own_blocks, shared_blocks, value_blocks;  // of 64
    uint32_t key_first, key_stride, value_first, value_stride, shared_first;
    uint32_t key_stages;
    float scale_log2;
    uint32_t one_pass;                                 // the row's maximum is bound_log2 * |temperature|
    float bound_log2, temp_coef;
    uint32_t temp_every;
    uint32_t *error_word;
};

uint32_t tc_smem_bytes(uint32_t q_blocks, uint32_t v_blocks, uint32_t key_stages) {
    return q_blocks * kRowBlock + key_stages * q_blocks * kKeyBlock + kValueStages * v_blocks * kKeyBlock + 2u * kRowBlock +
           kTail + 1024u;
}

__global__ void __launch_bounds__(kThreads, 1)
attend_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                 const __grid_constant__ CUtensorMap v_map, const __grid_constant__ CUtensorMap shared_map, const AttendTcParams p) {
    extern __shared__ uint8_t attend_tc_smem[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(attend_tc_smem) + 1023u) & ~(uintptr_t)1023u);
    const uint32_t qb = p.own_blocks + p.shared_blocks, vb = p.value_blocks;
    const uint32_t key_bytes = qb * kKeyBlock, value_bytes = vb * kKeyBlock;
    uint8_t *q_smem = smem, *k_smem = q_smem + qb * kRowBlock, *v_smem = k_smem + p.key_stages * key_bytes;
    uint8_t *p_smem = v_smem + kValueStages * value_bytes, *tail = p_smem + 2u * kRowBlock;
    uint64_t *bars = reinterpret_cast<uint64_t *>(tail);
    uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 4, *v_full = bars + 7, *v_empty = bars + 9;
    uint64_t *s_full = bars + 11, *s_free = bars + 13, *p_full = bars + 15, *p_free = bars + 16, *o_full = bars + 17;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 18);
    volatile uint32_t *abort_flag = tmem_slot + 1;
    float *exchange = reinterpret_cast<float *>(tail + 256u);  // [2][128]: what the two warps of a row tell each other

    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t head = blockIdx.x, key_head = head / (p.heads / p.key_heads);
    const uint32_t row0 = (gridDim.y - 1u - blockIdx.y) * 128u;  // late row blocks read the most keys: first
    const uint32_t last_row = min(p.m, row0 + 128u) - 1u;
    const uint32_t steps = (p.first_pos + last_row) / kKeys + 1u;

    if (tid == 0) {
        mbar_init(q_full, 1);
        for (uint32_t s = 0; s < kMaxKeyStages; ++s) {
            mbar_init(&k_full[s], 1);
            mbar_init(&k_empty[s], 1);
        }
        for (uint32_t s = 0; s < 2u; ++s) {
            mbar_init(&v_full[s], 1);
            mbar_init(&v_empty[s], 1);
            mbar_init(&s_full[s], 1);
            mbar_init(&s_free[s], kSoftmaxWarps);
        }
        mbar_init(p_full, kSoftmaxWarps);
        mbar_init(p_free, 1);
        mbar_init(o_full, 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == kSoftmaxWarps + 1u) tmem_alloc(tmem_slot, kTmemColumns);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    auto give_up = [&]() {
        *abort_flag = 1;
        atomicOr(p.error_word, kErrMbarTimeout);
    };

    if (warp == kSoftmaxWarps) {
        // ------------------------------------------------ tiles by TMA
        if (lane == 0) {
            mbar_arrive_expect_tx(q_full, qb * kRowBlock);
            for (uint32_t b = 0; b < qb; ++b)
                tma_load_2d(q_smem + b * kRowBlock, &q_map, (head * qb + b) * 64u, row0, q_full);
            uint32_t ks = 0, kph = 1, vs = 0, vph = 1;  // a fresh barrier passes a wait on parity 1
            bool ok = true;
            for (uint32_t pass = p.one_pass; pass < 2u && ok; ++pass) {
                for (uint32_t j = 0; j < steps && ok; ++j) {
                    const uint32_t page = (uint32_t)p.block_table[j], y = (page * p.key_heads + key_head) * kKeys;
                    if (!(ok = mbar_wait_bounded(&k_empty[ks], kph, abort_flag))) break;
                    uint8_t *dst = k_smem + ks * key_bytes;
                    mbar_arrive_expect_tx(&k_full[ks], key_bytes);
                    for (uint32_t b = 0; b < p.own_blocks; ++b)
                        tma_load_2d(dst + b * kKeyBlock, &k_map, p.key_first + head * p.key_stride + b * 64u, y, &k_full[ks]);
                    for (uint32_t b = 0; b < p.shared_blocks; ++b)
                        tma_load_2d(dst + (p.own_blocks + b) * kKeyBlock, &shared_map, p.shared_first + b * 64u, page * kKeys, &k_full[ks]);
                    if (++ks == p.key_stages) ks = 0, kph ^= 1u;
                    if (pass == 1u) {
                        if (!(ok = mbar_wait_bounded(&v_empty[vs], vph, abort_flag))) break;
                        mbar_arrive_expect_tx(&v_full[vs], value_bytes);
                        for (uint32_t b = 0; b < vb; ++b)
                            tma_load_2d(v_smem + vs * value_bytes + b * kKeyBlock, &v_map,
                                        p.value_first + head * p.value_stride + b * 64u, y, &v_full[vs]);
                        if (++vs == kValueStages) vs = 0, vph ^= 1u;
                    }
                }
            }
            if (!ok) give_up();
        }
    } else if (warp == kSoftmaxWarps + 1u) {
        // ------------------------------------------------ tensor-core issue
        if (lane == 0) {
            bool ok = mbar_wait_bounded(q_full, 0, abort_flag);
            uint32_t ks = 0, kph = 0, vs = 0, vph = 0, g = 0;  // g counts score tiles: buffer g & 1
            const uint32_t q_addr = smem_u32(q_smem), idesc_pv = kIdescPV | ((vb * 64u >> 3) << 17);
            auto scores = [&]() {
                const uint32_t b = g & 1u, use = g >> 1;
                ok = ok && mbar_wait_bounded(&k_full[ks], kph, abort_flag) &&
                     mbar_wait_bounded(&s_free[b], (use & 1u) ^ 1u, abort_flag);  // the softmax warps are done with use - 1
                if (!ok) return;
                tc_fence_after();
                const uint32_t k_addr = smem_u32(k_smem + ks * key_bytes);
                for (uint32_t blk = 0; blk < qb; ++blk)
#pragma unroll
                    for (uint32_t i = 0; i < 4u; ++i)  // 16 entries a step; 64 a block
                        umma_f16(tmem_base + b * kKeys, smem_desc_sw128(q_addr + blk * kRowBlock + i * 32u),
                                 smem_desc_sw128(k_addr + blk * kKeyBlock + i * 32u), kIdescS, (blk | i) != 0u ? 1u : 0u);
                umma_commit(&k_empty[ks]);
                umma_commit(&s_full[b]);
                if (++ks == p.key_stages) ks = 0, kph ^= 1u;
                ++g;
            };
            for (uint32_t j = 0; j < steps && ok && !p.one_pass; ++j) scores();
            const uint32_t hi_addr = smem_u32(p_smem), lo_addr = hi_addr + kRowBlock;
            for (uint32_t j = 0; j <= steps && ok; ++j) {
                if (j < steps) scores();  // step j is multiplied while step j - 1 is exponentiated
                if (j == 0u || !ok) continue;
                const uint32_t t = j - 1u;
                ok = mbar_wait_bounded(p_full, t & 1u, abort_flag) && mbar_wait_bounded(&v_full[vs], vph, abort_flag);
                if (!ok) break;
                tc_fence_after();
                const uint32_t v_addr = smem_u32(v_smem + vs * value_bytes);
#pragma unroll
                for (uint32_t i = 0; i < 4u; ++i) {  // 16 keys a step
                    const uint64_t vdesc = smem_desc_sw128_mn(v_addr + i * 2048u, kKeyBlock);
                    umma_f16(tmem_base + kOutColumn, smem_desc_sw128(hi_addr + i * 32u), vdesc, idesc_pv, (t | i) != 0u ? 1u : 0u);
                    umma_f16(tmem_base + kOutColumn, smem_desc_sw128(lo_addr + i * 32u), vdesc, idesc_pv, 1u);
                }
                umma_commit(&v_empty[vs]);
                umma_commit(p_free);
                if (++vs == kValueStages) vs = 0, vph ^= 1u;
            }
            if (!ok) give_up();
            umma_commit(o_full);  // also on the give-up path: the softmax warps wait on it
        }
    } else {
        // ------------------------------------------------ softmax: warps w and w + 4 share the 32 rows of lane group w & 3
        const uint32_t sub = warp & 3u, half = warp >> 2;
        const uint32_t r = 32u * sub + lane, row = row0 + r;
        const uint32_t pos = p.first_pos + min(row, p.m - 1u);  // last key this row may see
        const uint32_t lanes = (32u * sub) << 16, col0 = 32u * half;
        float mrow = -INFINITY;
        uint32_t g = 0;
        bool ok = true;
        for (uint32_t j = 0; j < steps && ok && !p.one_pass; ++j, ++g) {
            const uint32_t b = g & 1u;
            if (!(ok = mbar_wait_bounded(&s_full[b], (g >> 1) & 1u, abort_flag))) break;
            tc_fence_after();
            uint32_t v[32];
            tmem_ld_32x32(tmem_base + lanes + b * kKeys + col0, v);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_free[b]);
            const uint32_t key0 = j * kKeys + col0;
            float mx = -INFINITY;
            if (key0 + 31u <= pos) {  // the row sees the whole piece
#pragma unroll
                for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(v[i]));
            } else {
#pragma unroll
                for (int i = 0; i < 32; ++i)
                    if (key0 + i <= pos) mx = fmaxf(mx, __uint_as_float(v[i]));
            }
            mrow = fmaxf(mrow, mx * p.scale_log2);  // the scale is positive: it commutes with the maximum
        }
        if (p.one_pass) {
            mrow = p.bound_log2 * fabsf(query_temperature(pos, p.temp_coef, p.temp_every));
        } else {
            exchange[half * 128u + r] = mrow;
            named_bar_sync(1, kSoftmaxWarps * 32u);
            mrow = fmaxf(mrow, exchange[(half ^ 1u) * 128u + r]);
            named_bar_sync(1, kSoftmaxWarps * 32u);  // everybody has read: the words are free for the row sums
        }
        float l = 0.0f;
        uint8_t *p_hi = p_smem + r * 128u, *p_lo = p_hi + kRowBlock;
        for (uint32_t j = 0; j < steps && ok; ++j, ++g) {
            const uint32_t b = g & 1u;
            if (!(ok = mbar_wait_bounded(&s_full[b], (g >> 1) & 1u, abort_flag))) break;
            tc_fence_after();
            uint32_t v[32];
            tmem_ld_32x32(tmem_base + lanes + b * kKeys + col0, v);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_free[b]);
            uint32_t hi[16], lo[16];
            const uint32_t key0 = j * kKeys + col0;
            const bool whole = key0 + 31u <= pos;
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
                // exp2 of a non-positive argument by the hardware approximation: two units of an f32's last place
                float e0 = ex2_approx(fmaf(__uint_as_float(v[i]), p.scale_log2, -mrow));
                float e1 = ex2_approx(fmaf(__uint_as_float(v[i + 1]), p.scale_log2, -mrow));
                if (!whole) {
                    if (key0 + i > pos) e0 = 0.0f;
                    if (key0 + i + 1 > pos) e1 = 0.0f;
                }
                l += e0;
                l += e1;
                split_bf16x2(e0, e1, hi[i >> 1], lo[i >> 1]);
            }
            // the previous step's second product must have read P before it is overwritten
            if (!(ok = mbar_wait_bounded(p_free, (j & 1u) ^ 1u, abort_flag))) break;
            // 32 keys = four 16-byte chunks of the row's 128-byte line
#pragma unroll
            for (uint32_t q = 0; q < 4u; ++q) {
                const uint32_t at = ((half * 4u + q) ^ (r & 7u)) << 4;
                *reinterpret_cast<uint4 *>(p_hi + at) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
                *reinterpret_cast<uint4 *>(p_lo + at) = make_uint4(lo[4 * q], lo[4 * q + 1], lo[4 * q + 2], lo[4 * q + 3]);
            }
            proxy_fence_async();  // the tensor core reads shared memory through the async proxy
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
        }
        exchange[half * 128u + r] = l;
        named_bar_sync(1, kSoftmaxWarps * 32u);
        l = exchange[r] + exchange[128u + r];  // in key order
        const bool o_ok = mbar_wait_bounded(o_full, 0, abort_flag);
        if (!o_ok && lane == 0) atomicOr(p.error_word, kErrMbarTimeout);
        tc_fence_after();
        const float inv = l > 0.0f ? 1.0f / l : 0.0f;
        // ---- read-out of O: this warp's half of the columns
        uint16_t *dst = p.out + ((size_t)row * p.heads + head) * vb * 64u + half * vb * 32u;
        for (uint32_t c = 0; c < vb; ++c) {
            uint32_t v[32], packed[16];
            tmem_ld_32x32(tmem_base + lanes + kOutColumn + half * vb * 32u + c * 32u, v);
            if (row >= p.m || !o_ok || !ok) continue;
#pragma unroll
            for (int i = 0; i < 32; i += 2)
                packed[i >> 1] = f32x2_to_bf16x2(__uint_as_float(v[i]) * inv, __uint_as_float(v[i + 1]) * inv);
#pragma unroll
            for (int q = 0; q < 4; ++q)
                reinterpret_cast<uint4 *>(dst + 32u * c)[q] =
                    make_uint4(packed[4 * q], packed[4 * q + 1], packed[4 * q + 2], packed[4 * q + 3]);
        }
        if (!ok && lane == 0) give_up();
    }
    tc_fence_before();
    __syncthreads();
    if (warp == kSoftmaxWarps + 1u) {
        tc_fence_after();
        tmem_dealloc(tmem_base, kTmemColumns);
    }
}

constexpr uint32_t kSmemLimit = 227u * 1024u;

uint32_t stages_for(uint32_t key_blocks, uint32_t value_blocks) {
    for (uint32_t k = kMaxKeyStages; k >= 2u; --k)
        if (tc_smem_bytes(key_blocks, value_blocks, k) <= kSmemLimit) return k;
    return 0;
}

// Twice the bound is how far below it a score can lie; exp2 of that must stay well inside f32 and bf16.
constexpr float kMostBelowBound = 100.0f;

}  // namespace

bool attend_tc_supports(uint32_t key_blocks, uint32_t value_blocks) {
    return key_blocks && value_blocks && key_blocks <= kMaxBlocks && value_blocks <= kMaxBlocks &&
           stages_for(key_blocks, value_blocks) != 0 && encode_tiled() != nullptr;
}

stark_b200_status attend_tc_launch(const AttendTcArgs &a, cudaStream_t stream) {
    const uint32_t key_blocks = a.own_blocks + a.shared_blocks;
    if (!a.queries || !a.keys.base || !a.values.base || (a.shared_blocks && (!a.shared.base || a.key_heads != 1u)) || !a.out ||
        !a.block_table || a.m == 0 || a.ld_q % 8u || !(a.scale > 0.0f) || !a.key_heads || a.heads % a.key_heads ||
        (a.dim_bound > 0.0f && !a.temp_every))
        return STARK_B200_INVALID_ARGUMENT;
    if (!attend_tc_supports(key_blocks, a.value_blocks)) return STARK_B200_UNSUPPORTED;
    EncodeTiledFn encode = encode_tiled();
    const cuuint32_t elem[2] = {1u, 1u};
    CUtensorMap q_map, k_map, v_map, shared_map;
    auto make = [&](CUtensorMap *map, const void *base, uint64_t columns, uint64_t rows, uint64_t ld, uint32_t box_rows) {
        const cuuint64_t dims[2] = {columns, rows}, strides[1] = {ld * 2u};
        const cuuint32_t box[2] = {64u, box_rows};
        return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, elem,
                      CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                      CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
    };
    const AttendTile &shared = a.shared_blocks ? a.shared : a.keys;
    if (!make(&q_map, a.queries, (uint64_t)a.heads * key_blocks * 64u, a.m, a.ld_q, 128u) ||
        !make(&k_map, a.keys.base, a.keys.columns, a.keys.rows, a.keys.ld, kKeys) ||
        !make(&v_map, a.values.base, a.values.columns, a.values.rows, a.values.ld, kKeys) ||
        !make(&shared_map, shared.base, shared.columns, shared.rows, shared.ld, kKeys))
        return STARK_B200_DEVICE_FAILURE;
    AttendTcParams p{};
    p.out = a.out;
    p.block_table = a.block_table;
    p.m = a.m, p.first_pos = a.first_pos, p.heads = a.heads, p.key_heads = a.key_heads;
    p.own_blocks = a.own_blocks, p.shared_blocks = a.shared_blocks, p.value_blocks = a.value_blocks;
    p.key_first = a.keys.first, p.key_stride = a.keys.stride;
    p.value_first = a.values.first, p.value_stride = a.values.stride;
    p.shared_first = a.shared.first;
    p.key_stages = stages_for(key_blocks, a.value_blocks);
    p.scale_log2 = a.scale * kLog2e;
    if (a.dim_bound > 0.0f) {
        // the temperature moves one way with the position: its largest size is at the first or the last one
        const float most = std::max(fabsf(query_temperature(0, a.temp_coef, a.temp_every)),
                                    fabsf(query_temperature(a.first_pos + a.m - 1u, a.temp_coef, a.temp_every)));
        p.bound_log2 = p.scale_log2 * a.dim_bound;
        p.one_pass = 2.0f * p.bound_log2 * most <= kMostBelowBound ? 1u : 0u;
        p.temp_coef = a.temp_coef, p.temp_every = a.temp_every;
    }
    p.error_word = a.error_word;
    static SmemOptIn once;
    if (stark_b200_status st = ensure_dynamic_smem(attend_tc_kernel, (int)kSmemLimit, once)) return st;
    attend_tc_kernel<<<dim3(a.heads, (a.m + 127u) / 128u), kThreads, tc_smem_bytes(key_blocks, a.value_blocks, p.key_stages), stream>>>(
        q_map, k_map, v_map, shared_map, p);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

bool latent_prefill_tc_supports(const LatentShape &s) { return attend_tc_supports(s.q_head() / 64u, s.vdim_p / 64u); }

stark_b200_status latent_prefill_tc_launch(const LatentArgs &a, cudaStream_t stream) {
    if (!a.qd_b16 || a.cache_f32 || !a.cache || !a.expanded || !a.out_b16) return STARK_B200_INVALID_ARGUMENT;
    const LatentShape &s = a.s;
    const uint32_t rows = (a.first_pos + a.m + kPageTokens - 1u) / kPageTokens * kPageTokens;
    const uint32_t expanded = s.heads * (s.dim_p + s.vdim_p);
    AttendTcArgs t{};
    t.queries = static_cast<const uint16_t *>(a.qd);
    t.ld_q = a.ld_qd, t.heads = s.heads, t.key_heads = 1;
    t.keys = {a.expanded, expanded, rows, expanded, 0u, s.dim_p};
    t.values = {a.expanded, expanded, rows, expanded, s.heads * s.dim_p, s.vdim_p};
    t.shared = {static_cast<const uint16_t *>(a.cache), s.row(), a.num_blocks * kPageTokens, s.row(), s.rank_p, 0u};
    t.own_blocks = s.dim_p / 64u, t.shared_blocks = s.rot_p / 64u, t.value_blocks = s.vdim_p / 64u;
    t.block_table = a.block_table;
    t.first_pos = a.first_pos, t.m = a.m;
    t.scale = a.scale;
    t.out = static_cast<uint16_t *>(a.out);
    t.error_word = a.error_word;
    return attend_tc_launch(t, stream);
}

}  // namespace sb
