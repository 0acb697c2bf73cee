// The absorbed latent attention of one or a few rows over a bf16 cache, 16 heads at a time: what a decode step runs.
//
// All heads share the cached rows, so 16 heads are the M side of mma.sync.m16n8k16 tiles over a page of 64 keys.  A CTA
// owns 16 heads of one row over one span of pages:
//   page tile   [64 keys][row()] by TMA, 128-byte swizzled boxes of 64 columns (one or two tiles in flight).  Pages
//               before the last one were complete before this token began and are fetched before the wait on the
//               previous kernel; the last page holds the row that kernel appends
//   scores      the contraction index (latent + rotated part) is divided among the eight warps; a warp keeps its query
//               fragments in registers as bf16 hi + lo, the partial score tiles are added in shared memory
//   softmax     f32, running maximum and sum per head across the span's pages; weights as bf16 hi + lo
//   latents     the columns of the weighted sum are divided among the warps, accumulators stay in registers
// so scores and weights keep f32 accuracy against the bf16 cache.  A few spans' CTAs (four unless set otherwise) form a cluster and merge their
// (maximum, sum, weighted latents) through distributed shared memory, each taking a share of the columns; what is left for
// the value kernel to merge is one partial per cluster.  Every wait is bounded; a wait that runs out sets the error word.
#include <cuda.h>

#include "layered.cuh"
#include "layered_math.cuh"
#include "tc05.cuh"

namespace sb {

namespace {

constexpr uint32_t kWarps = 8, kThreads = kWarps * 32u, kHeads = 16;
constexpr uint32_t kBox = kPageTokens * 128u;      // 64 keys x 64 columns bf16
constexpr uint32_t kMaxSteps = 6;                  // 16-wide score steps per warp: rows up to 768 values
constexpr uint32_t kMaxBlocks = 2;                 // 64-wide latent blocks per warp
constexpr uint32_t kMaxCluster = 8;
constexpr uint32_t kScorePitch = 68, kWeightPitch = 72;
constexpr uint32_t kScoreBytes = kWarps * kHeads * kScorePitch * 4u, kWeightBytes = 2u * kHeads * kWeightPitch * 2u;

__device__ inline void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ inline void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr)
                 : "memory");
}
__device__ inline void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ inline void split(float x, float y, uint32_t &hi, uint32_t &lo) {
    hi = f32x2_to_bf16x2(x, y);
    lo = f32x2_to_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

__device__ inline void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// The address of a shared-memory word of this CTA in another CTA of the cluster.
__device__ inline uint32_t peer_smem(const void *p, uint32_t rank) {
    uint32_t a;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_u32(p)), "r"(rank));
    return a;
}
__device__ inline float peer_load(uint32_t addr) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
}
__device__ inline float4 peer_load4(uint32_t addr) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
    return v;
}

struct AttendParams {
    const float *queries;
    float *partials;
    const int32_t *block_table;
    const StepState *state;
    uint32_t first_pos, heads, latent_blocks, blocks;  // blocks of 64 columns: of the latent, of the whole row
    uint32_t splits, cluster;                          // partials a head leaves; CTAs (spans) merged into each
    uint32_t tiles;                                            // page tiles in flight: 1 or 2
    uint32_t *error_word;
};

// blockIdx: (span, group of 16 heads, row); BLOCKS: 64-wide latent blocks per warp
template <uint32_t BLOCKS>
__global__ void __launch_bounds__(kThreads, 1)
latent_attend_mma_kernel(const __grid_constant__ CUtensorMap map, const AttendParams p) {
    extern __shared__ uint8_t attend_tiles[];
    __shared__ float run_m[kHeads], run_l[kHeads], keep[kHeads];
    __shared__ uint64_t full[2];
    __shared__ uint32_t abort_flag;
    uint8_t *tile = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(attend_tiles) + 1023u) & ~(uintptr_t)1023u);
    const uint32_t tile_bytes = p.blocks * kBox, width = p.blocks * 64u, rank = p.latent_blocks * 64u;
    float *scores = reinterpret_cast<float *>(tile + p.tiles * tile_bytes);  // [warp][head][key]
    uint16_t *w_hi = reinterpret_cast<uint16_t *>(reinterpret_cast<uint8_t *>(scores) + kScoreBytes), *w_lo = w_hi + kHeads * kWeightPitch;
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t span_i = blockIdx.x, head0 = blockIdx.y * kHeads, row = blockIdx.z;
    // the step state does not change while a token's kernels run, except by its last one
    const uint32_t pos = p.state ? p.state->position : p.first_pos + row;
    const uint32_t pages = pos / kPageTokens + 1u, spans = p.splits * p.cluster, span = (pages + spans - 1u) / spans;
    const uint32_t lo = min(pages, span_i * span), hi = min(pages, lo + span);

    if (tid == 0) {
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        abort_flag = 0;
        mbar_fence_init();
    }
    if (tid < kHeads) run_m[tid] = -INFINITY, run_l[tid] = 0.0f;
    __syncthreads();
    auto fetch = [&](uint32_t page) {  // one thread
        const uint32_t slot = p.tiles == 2u ? (page - lo) & 1u : 0u;
        mbar_arrive_expect_tx(&full[slot], tile_bytes);
        const uint32_t y = (uint32_t)p.block_table[page] * kPageTokens;
        for (uint32_t b = 0; b < p.blocks; ++b) tma_load_2d(tile + slot * tile_bytes + b * kBox, &map, b * 64u, y, &full[slot]);
    };
    // fetched ahead of the wait: pages that cannot hold a row of this launch's predecessors
    const uint32_t first_new = p.state ? pages - 1u : 0u;
    uint32_t issued = lo;
    if (tid == 0)
        for (; issued < min(hi, lo + p.tiles) && issued < first_new; ++issued) fetch(issued);
    pdl_launch_dependents();
    pdl_wait();
    if (tid == 0)
        for (; issued < min(hi, lo + p.tiles); ++issued) fetch(issued);

    // ---- this warp's query fragments: steps warp, warp + 8, ... of 16 columns; rows are heads
    const uint32_t steps = p.blocks * 4u;
    uint32_t q_hi[kMaxSteps][4], q_lo[kMaxSteps][4];
#pragma unroll
    for (uint32_t i = 0; i < kMaxSteps; ++i) {
        const uint32_t s = warp + kWarps * i;
#pragma unroll
        for (uint32_t e = 0; e < 4u; ++e) {
            const uint32_t head = head0 + (lane >> 2) + (e & 1u) * 8u, col = s * 16u + (lane & 3u) * 2u + (e >> 1) * 8u;
            float2 v = make_float2(0.0f, 0.0f);
            if (s < steps && head < p.heads && lo < hi)
                v = *reinterpret_cast<const float2 *>(p.queries + ((size_t)row * p.heads + head) * width + col);
            split(v.x, v.y, q_hi[i][e], q_lo[i][e]);
        }
    }
    float out[BLOCKS][8][4];
#pragma unroll
    for (uint32_t b = 0; b < BLOCKS; ++b)
#pragma unroll
        for (uint32_t n = 0; n < 8u; ++n)
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) out[b][n][e] = 0.0f;

    const uint32_t mi = lane >> 3, mr = lane & 7u;  // ldmatrix: which 8 x 8 matrix this lane addresses, which row of it
    bool ok = true;
    for (uint32_t page = lo; page < hi && ok; ++page) {
        const uint32_t use = page - lo, slot = p.tiles == 2u ? use & 1u : 0u;
        const uint32_t phase = p.tiles == 2u ? (use >> 1) & 1u : use & 1u;
        ok = mbar_wait_bounded(&full[slot], phase, &abort_flag);
        ok = __syncthreads_and(ok);
        if (!ok) break;
        const uint32_t base = smem_u32(tile + slot * tile_bytes);
        float s[8][4];
#pragma unroll
        for (uint32_t n = 0; n < 8u; ++n)
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) s[n][e] = 0.0f;
#pragma unroll
        for (uint32_t i = 0; i < kMaxSteps; ++i) {
            const uint32_t st = warp + kWarps * i;
            if (st >= steps) break;
            const uint32_t box = base + (st >> 2) * kBox, chunk = (st & 3u) * 2u + (mi & 1u);
#pragma unroll
            for (uint32_t n2 = 0; n2 < 4u; ++n2) {  // 16 keys
                const uint32_t key = n2 * 16u + (mi >> 1) * 8u + mr;
                uint32_t b[4];
                ldmatrix_x4(b, box + key * 128u + ((chunk ^ (key & 7u)) << 4));
                mma_bf16(s[2u * n2], q_hi[i], b[0], b[1]);
                mma_bf16(s[2u * n2], q_lo[i], b[0], b[1]);
                mma_bf16(s[2u * n2 + 1u], q_hi[i], b[2], b[3]);
                mma_bf16(s[2u * n2 + 1u], q_lo[i], b[2], b[3]);
            }
        }
        float *mine = scores + warp * kHeads * kScorePitch;
#pragma unroll
        for (uint32_t n = 0; n < 8u; ++n) {
            const uint32_t col = n * 8u + (lane & 3u) * 2u, r = lane >> 2;
            *reinterpret_cast<float2 *>(mine + r * kScorePitch + col) = make_float2(s[n][0], s[n][1]);
            *reinterpret_cast<float2 *>(mine + (r + 8u) * kScorePitch + col) = make_float2(s[n][2], s[n][3]);
        }
        __syncthreads();
        {   // thread = (head, four keys)
            const uint32_t head = tid >> 4, key = (tid & 15u) * 4u;
            float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w) {
                const float4 a = *reinterpret_cast<const float4 *>(scores + (w * kHeads + head) * kScorePitch + key);
                v[0] += a.x, v[1] += a.y, v[2] += a.z, v[3] += a.w;
            }
            float top = -INFINITY;
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) {
                if (page * kPageTokens + key + e > pos) v[e] = -INFINITY;
                top = fmaxf(top, v[e]);
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
            const float before = run_m[head], now = fmaxf(before, top);
            float sum = 0.0f;
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) {
                v[e] = exp2f(v[e] - now);
                sum += v[e];
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            uint32_t h0, l0, h1, l1;
            split(v[0], v[1], h0, l0);
            split(v[2], v[3], h1, l1);
            *reinterpret_cast<uint2 *>(w_hi + head * kWeightPitch + key) = make_uint2(h0, h1);
            *reinterpret_cast<uint2 *>(w_lo + head * kWeightPitch + key) = make_uint2(l0, l1);
            __syncwarp();  // the sixteen threads of a head have read its running maximum
            if ((tid & 15u) == 0) {
                const float k = exp2f(before - now);  // 0 on the first page
                keep[head] = k;
                run_l[head] = run_l[head] * k + sum;
                run_m[head] = now;
            }
        }
        __syncthreads();
        const float k0 = keep[lane >> 2], k1 = keep[(lane >> 2) + 8u];
        if (page != lo) {
#pragma unroll
            for (uint32_t b = 0; b < BLOCKS; ++b)
#pragma unroll
                for (uint32_t n = 0; n < 8u; ++n) out[b][n][0] *= k0, out[b][n][1] *= k0, out[b][n][2] *= k1, out[b][n][3] *= k1;
        }
#pragma unroll
        for (uint32_t ks = 0; ks < 4u; ++ks) {  // 16 keys
            uint32_t ah[4], al[4];
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) {
                const uint32_t at = ((lane >> 2) + (e & 1u) * 8u) * kWeightPitch + ks * 16u + (lane & 3u) * 2u + (e >> 1) * 8u;
                ah[e] = *reinterpret_cast<const uint32_t *>(w_hi + at);
                al[e] = *reinterpret_cast<const uint32_t *>(w_lo + at);
            }
            const uint32_t key = ks * 16u + (mi & 1u) * 8u + mr;
#pragma unroll
            for (uint32_t b = 0; b < BLOCKS; ++b) {
                const uint32_t block = warp + kWarps * b;
                if (block >= p.latent_blocks) break;
                const uint32_t line = base + block * kBox + key * 128u;
#pragma unroll
                for (uint32_t n2 = 0; n2 < 4u; ++n2) {  // 16 columns
                    uint32_t v[4];
                    ldmatrix_x4_trans(v, line + (((n2 * 2u + (mi >> 1)) ^ (key & 7u)) << 4));
                    mma_bf16(out[b][2u * n2], ah, v[0], v[1]);
                    mma_bf16(out[b][2u * n2], al, v[0], v[1]);
                    mma_bf16(out[b][2u * n2 + 1u], ah, v[2], v[3]);
                    mma_bf16(out[b][2u * n2 + 1u], al, v[2], v[3]);
                }
            }
        }
        __syncthreads();  // everybody is through with this tile, the weights and the statistics
        if (tid == 0 && issued < hi) fetch(issued++);
    }
    if (!ok && tid == 0) {
        abort_flag = 1;
        atomicOr(p.error_word, kErrMbarTimeout);
    }
    // ---- merge within the cluster: this span's weighted latents and statistics into shared memory (the page tiles are
    // free), then every CTA forms its share of the columns over the cluster's spans
    float *state = reinterpret_cast<float *>(tile);  // [head][rank]
#pragma unroll
    for (uint32_t b = 0; b < BLOCKS; ++b) {
        const uint32_t block = warp + kWarps * b;
        if (block >= p.latent_blocks) break;
#pragma unroll
        for (uint32_t e = 0; e < 2u; ++e) {
            float *dst = state + ((lane >> 2) + 8u * e) * rank + block * 64u + (lane & 3u) * 2u;
#pragma unroll
            for (uint32_t n = 0; n < 8u; ++n) *reinterpret_cast<float2 *>(dst + n * 8u) = make_float2(out[b][n][2u * e], out[b][n][2u * e + 1u]);
        }
    }
    if (p.cluster > 1u) cluster_sync();
    else __syncthreads();
    const uint32_t me = span_i % p.cluster, split_i = span_i / p.cluster;
    // thread = (head, quads of this CTA's columns); an empty span's weight is 0 and its latents are zeros
    const uint32_t h = tid >> 4, head = head0 + h, quads = rank / 4u;
    float weight[kMaxCluster], top = -INFINITY, sum = 0.0f;
#pragma unroll
    for (uint32_t c = 0; c < kMaxCluster; ++c) {
        weight[c] = c < p.cluster ? peer_load(peer_smem(&run_m[h], c)) : -INFINITY;
        top = fmaxf(top, weight[c]);
    }
#pragma unroll
    for (uint32_t c = 0; c < kMaxCluster; ++c) {
        weight[c] = weight[c] == -INFINITY ? 0.0f : exp2f(weight[c] - top);
        if (c < p.cluster) sum = fmaf(weight[c], peer_load(peer_smem(&run_l[h], c)), sum);
    }
    if (head < p.heads) {
        float *dst = p.partials + (((size_t)row * p.heads + head) * p.splits + split_i) * (rank + 4u);
        if (me == 0u && (tid & 15u) == 0) {
            dst[0] = top;  // -infinity: no span of the cluster had a page
            dst[1] = sum;
        }
        for (uint32_t q = me + p.cluster * (tid & 15u); q < quads; q += 16u * p.cluster) {
            float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (uint32_t c = 0; c < kMaxCluster; ++c) {
                if (c >= p.cluster) break;
                const float4 x = peer_load4(peer_smem(state + h * rank + q * 4u, c));
                v.x = fmaf(weight[c], x.x, v.x), v.y = fmaf(weight[c], x.y, v.y);
                v.z = fmaf(weight[c], x.z, v.z), v.w = fmaf(weight[c], x.w, v.w);
            }
            *reinterpret_cast<float4 *>(dst + 4u + q * 4u) = v;
        }
    }
    if (p.cluster > 1u) cluster_sync();  // nobody leaves while another CTA may read its shared memory
}

uint32_t attend_smem(const LatentShape &s, uint32_t tiles) {
    return tiles * (s.row() / 64u) * kBox + kScoreBytes + kWeightBytes + 1024u;
}

}  // namespace

bool latent_attend_mma_supports(const LatentShape &s) {
    return s.row() / 16u <= kMaxSteps * kWarps && s.rank_p / 64u <= kMaxBlocks * kWarps && attend_smem(s, 1) <= 220u * 1024u &&
           encode_tiled() != nullptr;
}

stark_b200_status latent_attend_mma_launch(const LatentArgs &a, cudaStream_t stream) {
    if (!a.queries || !a.partials || a.cache_f32 || !a.cache || a.m == 0 || a.cluster == 0 || a.cluster > kMaxCluster)
        return STARK_B200_INVALID_ARGUMENT;
    const LatentShape &s = a.s;
    if (!latent_attend_mma_supports(s)) return STARK_B200_UNSUPPORTED;
    CUtensorMap map;
    const cuuint64_t dims[2] = {s.row(), (cuuint64_t)a.num_blocks * kPageTokens}, strides[1] = {(cuuint64_t)s.row() * 2u};
    const cuuint32_t box[2] = {64u, kPageTokens}, elem[2] = {1u, 1u};
    if (encode_tiled()(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, dims, strides, box, elem,
                       CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                       CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
        return STARK_B200_DEVICE_FAILURE;
    AttendParams p{a.queries, a.partials, a.block_table, a.state, a.first_pos, s.heads, s.rank_p / 64u, s.row() / 64u,
                   a.splits, a.cluster, attend_smem(s, 2) <= 220u * 1024u ? 2u : 1u, a.error_word};
    auto kernel = s.rank_p <= kWarps * 64u ? latent_attend_mma_kernel<1> : latent_attend_mma_kernel<2>;
    static SmemOptIn once[2];
    if (stark_b200_status st = ensure_dynamic_smem(kernel, 220 * 1024, once[s.rank_p <= kWarps * 64u ? 0 : 1])) return st;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(a.splits * a.cluster, (s.heads + kHeads - 1u) / kHeads, a.m);
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = attend_smem(s, p.tiles);
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = a.cluster;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.pdl ? 2 : 1;
    SB_CUDA(cudaLaunchKernelEx(&cfg, kernel, map, p));
    return STARK_B200_OK;
}

}  // namespace sb
