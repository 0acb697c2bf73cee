// One token of grouped-query attention with short convolutions, in one launch over a bf16 cache: what a decode step runs.
//
// A CTA owns up to 8 query heads of one key / value head over one span of pages:
//   pages       keys [64][dim_p] and values [64][vdim_p] by TMA, 128-byte swizzled boxes of 64 columns.  Every page was
//               complete before this token began except for the token's own row, so all of them are fetched before the wait
//               on the previous kernel, and the part of the convolutions that earlier tokens left is summed there too
//   own rows    after the wait every CTA forms its queries from the projected row (convolution, norm, temperature; bf16
//               hi + lo in shared memory).  The CTAs whose span ends with the token's own page also form its key and
//               value, patch them into the fetched tile, and store them, the values to mix with and the projected row for
//               later layers and positions
//   attention   eight warps, each 32 keys of every fourth page.  Keys are the M side of mma.sync.m16n8k16, heads the N side:
//               eight heads, or four whose hi and lo halves sit side by side (PACK), so that one product serves both.  f32
//               scores, running maximum and sum per head; the weights, hi + lo likewise, go from the score registers into
//               the second product (values transposed on the M side) through a register transpose
//   merge       warps through shared memory, the spans of a cluster through distributed shared memory, each CTA taking a
//               share of the columns; clusters beyond one leave partials for span_merge
// so scores and weights keep f32 accuracy against the bf16 cache.  Every wait is bounded; a wait that runs out sets the
// error word.
#include <cuda.h>

#include "device_math.cuh"
#include "layered.cuh"
#include "layered_math.cuh"
#include "tc05.cuh"

namespace sb {

namespace {

constexpr uint32_t kWarps = 8, kThreads = kWarps * 32u, kHeads = kGroupedHeadTile;
constexpr uint32_t kRound = 4;                 // pages read at a time, two warps each (two where tiles are so large)
constexpr uint32_t kBox = kPageTokens * 128u;  // 64 keys x 64 columns bf16
constexpr uint32_t kMaxBlocks = 4;             // heads up to 256 wide
constexpr uint32_t kMaxCluster = 8;
constexpr uint32_t kMaxSlots = 8;
constexpr uint32_t kSmemLimit = 220u * 1024u;  // dynamic; of 227 KB an SM has for its CTAs

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

// Ends the kernel's use of distributed shared memory: only that everybody has come this far matters, not what was written.
__device__ inline void cluster_leave() {
    asm volatile("barrier.cluster.arrive.relaxed.aligned;\n\tbarrier.cluster.wait.aligned;" ::: "memory");
}
// Over the lanes that hold the same columns of a product: lane / 4 varies.
__device__ inline float rows_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 4));
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 8));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 16));
}
__device__ inline float rows_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    v += __shfl_xor_sync(0xffffffffu, v, 8);
    return v + __shfl_xor_sync(0xffffffffu, v, 16);
}

// blockIdx: (span, head tile of a key / value head); VB: value blocks of 64 columns; PACK: at most four heads a tile
template <uint32_t VB, bool PACK>
__global__ void __launch_bounds__(kThreads, 1)
grouped_attend_mma_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map, const GroupedArgs a,
                          const uint32_t slots, const uint32_t tile_bytes) {
    extern __shared__ uint8_t grouped_smem[];
    __shared__ uint64_t full[kMaxSlots];
    __shared__ float warp_m[kWarps][kHeads], warp_l[kWarps][kHeads], run_m[kHeads], run_l[kHeads];
    __shared__ volatile uint32_t abort_flag;
    const GroupedShape &s = a.s;
    const uint32_t kb = s.dim_p / 64u, stage_bytes = (kb + VB) * kBox, q_pitch = s.dim_p + 8u;
    uint8_t *tile = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(grouped_smem) + 1023u) & ~(uintptr_t)1023u);
    constexpr uint32_t kLow = PACK ? 4u : 8u;  // rows of the lo halves behind those of the hi halves
    uint16_t *q_rows = reinterpret_cast<uint16_t *>(tile + tile_bytes);  // [2 * kLow][q_pitch]
    uint16_t *new_row = q_rows + 2u * kLow * q_pitch;                    // key, then value
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t head_tiles = (s.per() + kHeads - 1u) / kHeads;
    const uint32_t span_i = blockIdx.x, group = blockIdx.y / head_tiles, first_head = blockIdx.y % head_tiles * kHeads;
    const uint32_t heads = min(kHeads, s.per() - first_head), head0 = group * s.per() + first_head;
    // the step state does not change while a token's kernels run, except by its last one
    const uint32_t pos = a.state->position;
    const uint32_t pages = pos / kPageTokens + 1u, spans = a.splits * a.cluster, span = (pages + spans - 1u) / spans;
    const uint32_t lo = min(pages, span_i * span), n = min(pages, lo + span) - lo;
    const bool owner = n != 0u && lo + n == pages;  // this span ends with the page of the token's own row

    if (tid == 0) {
        for (uint32_t i = 0; i < slots; ++i) mbar_init(&full[i], 1);
        abort_flag = 0;
        mbar_fence_init();
    }
    __syncthreads();
    auto fetch = [&](uint32_t slot, uint32_t page) {  // one thread
        mbar_arrive_expect_tx(&full[slot], stage_bytes);
        const uint32_t y = (page * s.groups + group) * kPageTokens;
        uint8_t *dst = tile + slot * stage_bytes;
        for (uint32_t b = 0; b < kb; ++b) tma_load_2d(dst + b * kBox, &k_map, b * 64u, y, &full[slot]);
        for (uint32_t b = 0; b < VB; ++b) tma_load_2d(dst + (kb + b) * kBox, &v_map, b * 64u, y, &full[slot]);
    };
    if (tid == 0)
        for (uint32_t i = 0; i < min(n, slots); ++i) fetch(i, (uint32_t)a.block_table[lo + i]);

    // ---- queries of this CTA's heads, and the token's own key and value where they are needed.  A unit is one head of the
    // three, a warp's; units 0 and 1 are the key and the value, which take the longest way.
    const uint32_t taps = a.conv.taps, width = s.width(), recent_rows = a.conv.recent_rows();
    const uint32_t in_page = pos % kPageTokens, last_page = (uint32_t)a.block_table[pages - 1u];
    const bool tail = in_page + taps > kPageTokens;  // one of the page's last taps - 1 positions
    auto unit_blocks = [&](uint32_t unit) {          // 0: nothing to do
        if (n == 0u || (unit < 2u && !owner) || unit >= heads + 2u) return 0u;
        return (unit == 1u ? s.vdim_p : s.dim_p) / 64u;
    };
    auto unit_col = [&](uint32_t unit) {
        return (unit >= 2u ? (head0 + unit - 2u) * s.dim_p : (unit == 0u ? s.key_col() + group * s.dim_p : s.value_col() + group * s.vdim_p)) +
               lane * 2u;
    };
    float2 v[kMaxBlocks], newest[kMaxBlocks];  // the convolution's sum; its weights for the token's own row
    auto past = [&](uint32_t unit) {           // the part of the sum that earlier tokens left, and the weights
        const uint32_t blocks = unit_blocks(unit), col = unit_col(unit);
        const float *w = a.conv.w + col;
        const uint16_t *recent = reinterpret_cast<const uint16_t *>(a.conv.recent) + col;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            v[b] = make_float2(0.0f, 0.0f);
            if (b < blocks) newest[b] = load_pair(w + (size_t)(taps - 1u) * width + b * 64u);
        }
        for (uint32_t j0 = 0; j0 + 1u < taps; j0 += 4u) {
            float2 x[kMaxBlocks][4], f[kMaxBlocks][4];
#pragma unroll
            for (uint32_t i = 0; i < 4u; ++i) {
                const uint32_t j = j0 + i, back = taps - 1u - j;
                const bool in = j + 1u < taps && back <= pos;  // nothing precedes the first token
#pragma unroll
                for (uint32_t b = 0; b < kMaxBlocks; ++b) {
                    x[b][i] = f[b][i] = make_float2(0.0f, 0.0f);
                    if (in && b < blocks) {
                        x[b][i] = load_pair(recent + (size_t)((pos - back) % recent_rows) * width + b * 64u);
                        f[b][i] = load_pair(w + (size_t)j * width + b * 64u);
                    }
                }
            }
#pragma unroll
            for (uint32_t i = 0; i < 4u; ++i)
#pragma unroll
                for (uint32_t b = 0; b < kMaxBlocks; ++b) {
                    v[b].x = fmaf(f[b][i].x, x[b][i].x, v[b].x);
                    v[b].y = fmaf(f[b][i].y, x[b][i].y, v[b].y);
                }
        }
    };
    past(warp);  // nothing of this depends on the kernels before
    const float q_factor = query_temperature(pos, a.temp_coef, a.temp_every) * (a.scale * kLog2e);
    for (uint32_t i = heads * q_pitch + tid; i < kLow * q_pitch; i += kThreads) q_rows[i] = q_rows[kLow * q_pitch + i] = 0u;
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t unit = warp; unit < heads + 2u; unit += kWarps) {
        if (unit != warp) past(unit);
        const bool is_k = unit == 0u, is_v = unit == 1u, is_q = unit >= 2u;
        const uint32_t h = unit - 2u, blocks = unit_blocks(unit), col = unit_col(unit);
        if (blocks == 0u) continue;
        const float *u = reinterpret_cast<const float *>(a.u) + col;
        float2 x[kMaxBlocks], mixed[kMaxBlocks];
        float sum = 0.0f;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b)
            if (b < blocks) x[b] = load_pair(u + b * 64u);
        float *first = a.first_values + group * s.vdim;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            if (b >= blocks) break;
            const float2 f = newest[b];
            mixed[b] = v[b];
            mixed[b].x = fmaf(f.x, x[b].x, mixed[b].x), mixed[b].y = fmaf(f.y, x[b].y, mixed[b].y);
            sum += mixed[b].x * mixed[b].x + mixed[b].y * mixed[b].y;
        }
        float factor = 1.0f;
        if (!is_v) factor = inverse_rms(warp_sum(sum), s.dim, a.eps);
        if (is_q) factor *= q_factor;
        const bool stores = owner && (is_q || first_head == 0u);  // one CTA per stored value
        uint16_t *dst = reinterpret_cast<uint16_t *>(is_k ? a.keys : a.values) +
                        (((size_t)last_page * s.groups + group) * kPageTokens + in_page) * (is_v ? s.vdim_p : s.dim_p) + lane * 2u;
        uint16_t *row = new_row + (is_k ? 0u : s.dim_p) + lane * 2u;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            if (b >= blocks) break;
            float2 o = make_float2(mixed[b].x * factor, mixed[b].y * factor);
            if (is_q) {
                uint32_t hi, lo2;
                split_bf16x2(o.x, o.y, hi, lo2);
                *reinterpret_cast<uint32_t *>(q_rows + h * q_pitch + lane * 2u + b * 64u) = hi;
                *reinterpret_cast<uint32_t *>(q_rows + (kLow + h) * q_pitch + lane * 2u + b * 64u) = lo2;
            } else {
                if (is_v && a.mix == kMixFirst && stores) keep_first_values(first, lane * 2u + b * 64u, s.vdim, o);
                if (is_v && a.mix == kMixShare) o = mix_values(first, lane * 2u + b * 64u, s.vdim, o, a.share);
                store_pair(row + b * 64u, o);
                if (stores) store_pair(dst + b * 64u, o);
            }
        }
        if (stores && taps > 1u) {  // the projected row itself, where a later position's convolution will look for it
            uint16_t *recent = reinterpret_cast<uint16_t *>(a.conv.recent) + (size_t)(pos % recent_rows) * width + col;
            uint16_t *tails = reinterpret_cast<uint16_t *>(a.conv.tails) +
                              ((size_t)last_page * (taps - 1u) + (tail ? in_page + taps - 1u - kPageTokens : 0u)) * width + col;
#pragma unroll
            for (uint32_t b = 0; b < kMaxBlocks; ++b) {
                if (b >= blocks) break;
                store_pair(recent + b * 64u, x[b]);
                if (tail) store_pair(tails + b * 64u, x[b]);
            }
        }
    }
    __syncthreads();

    // ---- attention: warps 2j and 2j + 1 take pages j, j + 4, ... of the span, half the keys each
    const uint32_t key0 = (warp & 1u) * 32u;
    const uint32_t mi = lane >> 3, mr = lane & 7u;  // ldmatrix: which 8 x 8 matrix this lane addresses, which row of it
    const uint32_t col = (lane & 3u) * 2u;          // this lane's columns of a product: two heads (PACK: modulo 4)
    uint32_t qf[kMaxBlocks * 4u][2], ql[PACK ? 1u : kMaxBlocks * 4u][2];
#pragma unroll
    for (uint32_t i = 0; i < kMaxBlocks * 4u; ++i) {
        if (i >= kb * 4u) break;
        const uint16_t *src = q_rows + (lane >> 2) * q_pitch + i * 16u + col;
        qf[i][0] = *reinterpret_cast<const uint32_t *>(src), qf[i][1] = *reinterpret_cast<const uint32_t *>(src + 8u);
        if constexpr (!PACK) {
            ql[i][0] = *reinterpret_cast<const uint32_t *>(src + kLow * q_pitch);
            ql[i][1] = *reinterpret_cast<const uint32_t *>(src + kLow * q_pitch + 8u);
        }
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f}, out[VB * 4u][4];  // l: this lane's keys only
#pragma unroll
    for (uint32_t i = 0; i < VB * 4u; ++i)
#pragma unroll
        for (uint32_t e = 0; e < 4u; ++e) out[i][e] = 0.0f;
    auto ldm = [](uint32_t (&r)[4], uint32_t addr) {
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                     : "r"(addr)
                     : "memory");
    };
    auto ldm_trans = [](uint32_t (&r)[4], uint32_t addr) {
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                     : "r"(addr)
                     : "memory");
    };
    const uint32_t round = min(kRound, slots);
    uint32_t slot0 = 0, phase0 = 0, fetched = min(n, slots);  // slot and phase of page i0; pages asked for (thread 0)
    for (uint32_t i0 = 0; i0 < n; i0 += round) {
        const uint32_t i = i0 + (warp >> 1);
        const bool wraps = slot0 + (warp >> 1) >= slots;
        const uint32_t slot = slot0 + (warp >> 1) - (wraps ? slots : 0u), phase = phase0 ^ (wraps ? 1u : 0u);
        uint32_t coming[kRound];  // pages that take the places of those read now
        if (tid == 0)
#pragma unroll
            for (uint32_t j = 0; j < kRound; ++j)
                coming[j] = j < round && i0 + slots + j < n ? (uint32_t)a.block_table[lo + i0 + slots + j] : UINT32_MAX;
        bool ok = i < n && (warp >> 1) < round && (lo + i) * kPageTokens + key0 <= pos;  // something to see; the same for the whole warp
        if (ok && !(ok = mbar_wait_bounded(&full[slot], phase, &abort_flag))) {
            abort_flag = 1;
            if (lane == 0) atomicOr(a.error_word, kErrMbarTimeout);
        }
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            uint8_t *stage = tile + slot * stage_bytes;
            const uint32_t row = pos % kPageTokens;
            if (lo + i + 1u == pages && (row & ~31u) == key0) {  // this warp's keys include the token's own
                const uint4 *src = reinterpret_cast<const uint4 *>(new_row);
                for (uint32_t c = lane; c < (kb + VB) * 8u; c += 32u)
                    *reinterpret_cast<uint4 *>(stage + (c >> 3) * kBox + row * 128u + (((c & 7u) ^ (row & 7u)) << 4)) = src[c];
                __syncwarp();
            }
            const uint32_t base = smem_u32(stage);
            float sc[2][4] = {}, low[2][4] = {};  // [16 keys][keys lane / 4 and + 8, two heads each]
            const uint32_t key = key0 + (mi & 1u) * 8u + mr, key_line = base + key * 128u;
#pragma unroll
            for (uint32_t b = 0; b < kMaxBlocks; ++b) {
                if (b >= kb) break;
#pragma unroll
                for (uint32_t k16 = 0; k16 < 4u; ++k16) {  // 16 columns
#pragma unroll
                    for (uint32_t g = 0; g < 2u; ++g) {    // 16 keys
                        uint32_t kf[4];
                        ldm(kf, key_line + g * 2048u + b * kBox + (((k16 * 2u + (mi >> 1)) ^ (key & 7u)) << 4));
                        mma_m16n8k16_bf16(sc[g], kf[0], kf[1], kf[2], kf[3], qf[b * 4u + k16][0], qf[b * 4u + k16][1]);
                        if constexpr (!PACK)
                            mma_m16n8k16_bf16(low[g], kf[0], kf[1], kf[2], kf[3], ql[b * 4u + k16][0], ql[b * 4u + k16][1]);
                    }
                }
            }
            const uint32_t first_key = (lo + i) * kPageTokens + key0 + (lane >> 2);
            float keep[2];
            uint32_t pf[2][2], pl[2][2];  // weights as the second product wants them: [16 keys][8 of them]
            {
                float w[2][4], top[2] = {-INFINITY, -INFINITY};
#pragma unroll
                for (uint32_t g = 0; g < 2u; ++g)
#pragma unroll
                    for (uint32_t e = 0; e < 4u; ++e) {
                        w[g][e] = sc[g][e] + (PACK ? __shfl_xor_sync(0xffffffffu, sc[g][e], 2) : low[g][e]);
                        if (first_key + g * 16u + (e >> 1) * 8u > pos) w[g][e] = -INFINITY;
                        top[e & 1u] = fmaxf(top[e & 1u], w[g][e]);
                    }
#pragma unroll
                for (uint32_t e = 0; e < 2u; ++e) {
                    top[e] = fmaxf(m[e], rows_max(top[e]));
                    keep[e] = exp2f(m[e] - top[e]);  // 0 at first
                    m[e] = top[e];
                    l[e] *= keep[e];
                }
#pragma unroll
                for (uint32_t g = 0; g < 2u; ++g)
#pragma unroll
                    for (uint32_t e = 0; e < 4u; e += 2u) {
                        const float w0 = exp2f(w[g][e] - top[0]), w1 = exp2f(w[g][e + 1u] - top[1]);
                        l[0] += w0, l[1] += w1;
                        uint32_t hi, lo2;
                        split_bf16x2(w0, w1, hi, lo2);
                        if constexpr (PACK) {
                            pf[g][e >> 1] = movmatrix_trans(col < 4u ? hi : lo2);
                        } else {
                            pf[g][e >> 1] = movmatrix_trans(hi);
                            pl[g][e >> 1] = movmatrix_trans(lo2);
                        }
                    }
            }
            const uint32_t vkey = key0 + (mi >> 1) * 8u + mr, value_line = base + kb * kBox + vkey * 128u;
#pragma unroll
            for (uint32_t v16 = 0; v16 < VB * 4u; ++v16) {  // 16 columns
                float(&o)[4] = out[v16];
                o[0] *= keep[0], o[1] *= keep[1], o[2] *= keep[0], o[3] *= keep[1];
#pragma unroll
                for (uint32_t g = 0; g < 2u; ++g) {
                    uint32_t vf[4];
                    ldm_trans(vf, value_line + g * 2048u + (v16 >> 2) * kBox + ((((v16 & 3u) * 2u + (mi & 1u)) ^ (vkey & 7u)) << 4));
                    mma_m16n8k16_bf16(o, vf[0], vf[1], vf[2], vf[3], pf[g][0], pf[g][1]);
                    if constexpr (!PACK) mma_m16n8k16_bf16(o, vf[0], vf[1], vf[2], vf[3], pl[g][0], pl[g][1]);
                }
            }
        }
        if (i0 + slots < n) {
            __syncthreads();
            if (tid == 0) {
                uint32_t into = slot0;
#pragma unroll
                for (uint32_t j = 0; j < kRound; ++j) {
                    if (coming[j] != UINT32_MAX && !abort_flag) fetch(into, coming[j]), ++fetched;
                    if (++into == slots) into = 0u;
                }
            }
        }
        if ((slot0 += round) >= slots) slot0 -= slots, phase0 ^= 1u;
    }

    if (tid == 0 && abort_flag) {  // what is still on its way must not land in the words below
        const uint32_t go_on = 0u;
        for (uint32_t i = fetched - min(fetched, slots); i < fetched; ++i) mbar_wait_bounded(&full[i % slots], (i / slots) & 1u, &go_on);
    }

    // ---- merge of the warps: statistics, then weighted values, rows pitch apart
    const uint32_t pitch = s.vdim_p + 8u;
    float *state = reinterpret_cast<float *>(tile);  // [warp][head][pitch]; the sum ends up in warp 0's part
#pragma unroll
    for (uint32_t e = 0; e < 2u; ++e) {
        l[e] = rows_sum(l[e]);
        if (lane < (PACK ? 2u : 4u)) warp_m[warp][col + e] = m[e], warp_l[warp][col + e] = l[e];
    }
    __syncthreads();  // everybody is through with the tiles as well
    {
        float mine[2];
#pragma unroll
        for (uint32_t e = 0; e < 2u; ++e) {
            const uint32_t h = (PACK ? col & 2u : col) + e;
            float top = -INFINITY;
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w) top = fmaxf(top, warp_m[w][h]);
            mine[e] = m[e] == -INFINITY ? 0.0f : exp2f(m[e] - top);
        }
#pragma unroll
        for (uint32_t v16 = 0; v16 < VB * 4u; ++v16)
#pragma unroll
            for (uint32_t e = 0; e < 4u; ++e) {  // columns lane / 4 and + 8 of 16, two heads each
                float o = out[v16][e] * mine[e & 1u];
                if constexpr (PACK) o += __shfl_xor_sync(0xffffffffu, o, 2);
                const uint32_t h = col + (e & 1u);
                if (h < heads) state[((size_t)warp * heads + h) * pitch + v16 * 16u + (e >> 1) * 8u + (lane >> 2)] = o;
            }
        if (tid < heads) {
            float top = -INFINITY, sum = 0.0f;
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w) top = fmaxf(top, warp_m[w][tid]);
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w)
                if (warp_m[w][tid] != -INFINITY) sum = fmaf(exp2f(warp_m[w][tid] - top), warp_l[w][tid], sum);
            run_m[tid] = top, run_l[tid] = sum;
        }
    }
    __syncthreads();
    const uint32_t quads = s.vdim_p / 4u;
    for (uint32_t t = tid; t < heads * quads; t += kThreads) {
        float *at = state + (t / quads) * pitch + t % quads * 4u;
        float4 v = *reinterpret_cast<const float4 *>(at);
#pragma unroll
        for (uint32_t w = 1; w < kWarps; ++w) {
            const float4 x = *reinterpret_cast<const float4 *>(at + (size_t)w * heads * pitch);
            v.x += x.x, v.y += x.y, v.z += x.z, v.w += x.w;
        }
        *reinterpret_cast<float4 *>(at) = v;
    }
    // ---- merge of the cluster's spans, a share of the columns each; an empty span weighs 0
    if (a.cluster > 1u) cluster_sync();
    else __syncthreads();
    const uint32_t me = span_i % a.cluster, split_i = span_i / a.cluster;
    for (uint32_t t = me + a.cluster * tid; t < heads * quads; t += a.cluster * kThreads) {
        const uint32_t h = t / quads, q = t % quads;
        float weight[kMaxCluster], sums[kMaxCluster], top = -INFINITY, sum = 0.0f;
        float4 x[kMaxCluster], v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (uint32_t c = 0; c < kMaxCluster; ++c) {  // all on their way before the first is used
            const uint32_t from = c < a.cluster ? c : 0u;
            weight[c] = peer_load(peer_smem(&run_m[h], from));
            sums[c] = peer_load(peer_smem(&run_l[h], from));
            x[c] = peer_load4(peer_smem(state + h * pitch + q * 4u, from));
        }
#pragma unroll
        for (uint32_t c = 0; c < kMaxCluster; ++c) {
            if (c >= a.cluster) weight[c] = -INFINITY;
            top = fmaxf(top, weight[c]);
        }
#pragma unroll
        for (uint32_t c = 0; c < kMaxCluster; ++c) {
            const float k = weight[c] == -INFINITY ? 0.0f : exp2f(weight[c] - top);
            sum = fmaf(k, sums[c], sum);
            v.x = fmaf(k, x[c].x, v.x), v.y = fmaf(k, x[c].y, v.y), v.z = fmaf(k, x[c].z, v.z), v.w = fmaf(k, x[c].w, v.w);
        }
        if (a.splits == 1u) {
            const float inv = 1.0f / sum;
            *reinterpret_cast<float4 *>(a.out + (size_t)(head0 + h) * s.vdim_p + q * 4u) = make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv);
        } else {
            float *dst = a.partials + ((size_t)(head0 + h) * a.splits + split_i) * (s.vdim_p + 4u);
            if (q == 0u) dst[0] = top, dst[1] = sum;  // -infinity: no span of the cluster had a page
            *reinterpret_cast<float4 *>(dst + 4u + q * 4u) = v;
        }
    }
    if (a.cluster > 1u) cluster_leave();  // nobody leaves while another CTA may read its shared memory
}

struct Layout {
    uint32_t slots, tile_bytes, smem;
};
// `beside`: shared memory of an SM to leave for the CTAs of the kernels around this one.
Layout layout_of(const GroupedShape &s, uint32_t beside) {
    const uint32_t stage = (s.dim_p + s.vdim_p) / 64u * kBox, heads = std::min(kHeads, s.per());
    const uint32_t rows = 2u * (heads <= 4u ? 4u : 8u) * (s.dim_p + 8u) * 2u + (s.dim_p + s.vdim_p) * 2u + 1024u;
    const uint32_t room = kSmemLimit - std::min(beside, kSmemLimit / 2u);
    Layout l{};
    l.slots = std::min(kMaxSlots, std::max(2u, (room - std::min(rows, room)) / stage));
    if (l.slots < kRound) l.slots = 2u;
    l.tile_bytes = std::max(l.slots * stage, kWarps * heads * (s.vdim_p + 8u) * 4u);
    l.tile_bytes = (l.tile_bytes + 127u) & ~127u;
    l.smem = l.tile_bytes + rows;
    return l;
}

using Kernel = void (*)(const CUtensorMap, const CUtensorMap, const GroupedArgs, uint32_t, uint32_t);
template <bool PACK>
Kernel kernel_of(uint32_t value_blocks) {
    return value_blocks == 1u ? grouped_attend_mma_kernel<1, PACK>
                              : (value_blocks == 2u ? grouped_attend_mma_kernel<2, PACK>
                                                    : (value_blocks == 3u ? grouped_attend_mma_kernel<3, PACK> : grouped_attend_mma_kernel<4, PACK>));
}

}  // namespace

bool grouped_attend_mma_supports(const GroupedShape &s) {
    return s.dim_p <= kMaxBlocks * 64u && s.vdim_p <= kMaxBlocks * 64u && layout_of(s, kSmemLimit).smem <= kSmemLimit && encode_tiled() != nullptr;
}

stark_b200_status grouped_attend_mma_launch(const GroupedArgs &a, cudaStream_t stream) {
    const GroupedShape &s = a.s;
    if (!grouped_shape_supported(s, a.conv.taps) || !grouped_attend_mma_supports(s)) return STARK_B200_UNSUPPORTED;
    if (!a.u || a.u_b16 || a.cache_f32 || !a.conv.w || !a.conv.recent || !a.conv.tails || !a.keys || !a.values || !a.block_table ||
        !a.state || a.m != 1u || !a.temp_every || (a.mix != kMixNone && !a.first_values) || a.cluster == 0 ||
        a.cluster > kMaxCluster || (a.cluster & (a.cluster - 1u)) || a.splits == 0 || a.splits > kMaxSplits ||
        (a.splits == 1u ? !a.out : !a.partials))
        return STARK_B200_INVALID_ARGUMENT;
    const bool pack = s.per() <= 4u;
    const Kernel kernel = pack ? kernel_of<true>(s.vdim_p / 64u) : kernel_of<false>(s.vdim_p / 64u);
    static SmemOptIn once[2][kMaxBlocks];
    if (stark_b200_status st = ensure_dynamic_smem(kernel, (int)kSmemLimit, once[pack][s.vdim_p / 64u - 1u])) return st;
    CUtensorMap k_map, v_map;
    auto make = [&](CUtensorMap *map, void *base, uint32_t columns) {
        const cuuint64_t dims[2] = {columns, (cuuint64_t)a.num_blocks * s.groups * kPageTokens}, strides[1] = {(cuuint64_t)columns * 2u};
        const cuuint32_t box[2] = {64u, kPageTokens}, elem[2] = {1u, 1u};
        return encode_tiled()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, base, dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) ==
               CUDA_SUCCESS;
    };
    if (!make(&k_map, a.keys, s.dim_p) || !make(&v_map, a.values, s.vdim_p)) return STARK_B200_DEVICE_FAILURE;
    const Layout l = layout_of(s, a.beside_smem);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(a.splits * a.cluster, s.groups * ((s.per() + kHeads - 1u) / kHeads));
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = l.smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = a.cluster;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.pdl ? 2 : 1;
    SB_CUDA(cudaLaunchKernelEx(&cfg, kernel, k_map, v_map, a, l.slots, l.tile_bytes));
    return STARK_B200_OK;
}

}  // namespace sb
