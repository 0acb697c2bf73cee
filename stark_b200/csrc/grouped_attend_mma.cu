// One token of grouped-query attention with short convolutions, in one launch over a bf16 cache: what a decode step runs.
//
// A CTA owns up to 16 query heads of one key / value head (the M side of mma.sync.m16n8k16) over one span of pages:
//   pages       keys [64][dim_p] and values [64][vdim_p] by TMA, 128-byte swizzled boxes of 64 columns.  Every page was
//               complete before this token began except for the token's own row, so all of them are fetched before the wait
//               on the previous kernel
//   own rows    after the wait every CTA forms its queries from the projected row and the recent ones (convolution, norm,
//               temperature; bf16 hi + lo in shared memory).  The CTAs whose span ends with the token's own page also form
//               its key and value, patch them into the fetched tile, and store them, the mixed-from values and the
//               projected row for later positions
//   attention   eight warps, each 16 keys of a page of its own pair (even and odd pages): f32 scores, running maximum and
//               sum per head, weights as bf16 hi + lo straight from the score registers, weighted values in registers
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

constexpr uint32_t kWarps = 8, kThreads = kWarps * 32u, kHeads = 16;
constexpr uint32_t kBox = kPageTokens * 128u;  // 64 keys x 64 columns bf16
constexpr uint32_t kMaxBlocks = 4;             // heads up to 256 wide
constexpr uint32_t kMaxCluster = 8;
constexpr uint32_t kMaxSlots = 8;
constexpr uint32_t kTileBudget = 128u * 1024u, kSmemLimit = 220u * 1024u;

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

__device__ inline float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ inline float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

// blockIdx: (span, head tile of a key / value head); VB: value blocks of 64 columns
template <uint32_t VB>
__global__ void __launch_bounds__(kThreads, 1)
grouped_attend_mma_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map, const GroupedArgs a,
                          const uint32_t slots, const uint32_t tile_bytes) {
    extern __shared__ uint8_t grouped_smem[];
    __shared__ uint64_t full[kMaxSlots];
    __shared__ float warp_m[kWarps][kHeads], warp_l[kWarps][kHeads], run_m[kHeads], run_l[kHeads];
    __shared__ uint32_t abort_flag;
    const GroupedShape &s = a.s;
    const uint32_t kb = s.dim_p / 64u, stage_bytes = (kb + VB) * kBox, q_pitch = s.dim_p + 8u;
    uint8_t *tile = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(grouped_smem) + 1023u) & ~(uintptr_t)1023u);
    uint16_t *q_hi = reinterpret_cast<uint16_t *>(tile + tile_bytes), *q_lo = q_hi + kHeads * q_pitch;  // [head][q_pitch]
    uint16_t *new_row = q_lo + kHeads * q_pitch;                                                       // key, then value
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
    auto fetch = [&](uint32_t i) {  // one thread
        const uint32_t slot = i % slots;
        mbar_arrive_expect_tx(&full[slot], stage_bytes);
        const uint32_t y = ((uint32_t)a.block_table[lo + i] * s.groups + group) * kPageTokens;
        uint8_t *dst = tile + slot * stage_bytes;
        for (uint32_t b = 0; b < kb; ++b) tma_load_2d(dst + b * kBox, &k_map, b * 64u, y, &full[slot]);
        for (uint32_t b = 0; b < VB; ++b) tma_load_2d(dst + (kb + b) * kBox, &v_map, b * 64u, y, &full[slot]);
    };
    if (tid == 0)
        for (uint32_t i = 0; i < min(n, slots); ++i) fetch(i);

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
                const bool in = j + 1u < taps && back <= pos;  // zeros before the sequence's start
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
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t unit = warp; unit < kHeads + 2u; unit += kWarps) {
        if (unit != warp) past(unit);
        const bool is_k = unit == 0u, is_v = unit == 1u, is_q = unit >= 2u;
        const uint32_t h = unit - 2u, blocks = unit_blocks(unit), col = unit_col(unit);
        if (is_q && h >= heads) {
            for (uint32_t c = lane * 2u; c < s.dim_p; c += 64u) {
                *reinterpret_cast<uint32_t *>(q_hi + h * q_pitch + c) = 0u;
                *reinterpret_cast<uint32_t *>(q_lo + h * q_pitch + c) = 0u;
            }
        }
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
        if (is_q) factor *= query_temperature(pos, a.temp_coef, a.temp_every) * (a.scale * kLog2e);
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
                *reinterpret_cast<uint32_t *>(q_hi + h * q_pitch + lane * 2u + b * 64u) = hi;
                *reinterpret_cast<uint32_t *>(q_lo + h * q_pitch + lane * 2u + b * 64u) = lo2;
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

    // ---- attention: warps 0-3 take the span's even pages, 4-7 the odd ones, 16 keys each
    const uint32_t half = warp >> 2, key0 = (warp & 3u) * 16u;
    const uint32_t mi = lane >> 3, mr = lane & 7u;  // ldmatrix: which 8 x 8 matrix this lane addresses, which row of it
    const uint32_t q_at = smem_u32(q_hi) + (((lane & 7u) + ((lane >> 3) & 1u) * 8u) * q_pitch + (lane >> 4) * 8u) * 2u;
    const uint32_t q_lo_at = q_at + kHeads * q_pitch * 2u;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f}, out[VB * 8u][4];
#pragma unroll
    for (uint32_t i = 0; i < VB * 8u; ++i)
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
    for (uint32_t i0 = 0; i0 < n; i0 += 2u) {
        const uint32_t i = i0 + half;
        bool ok = i < n;
        if (ok && !(ok = mbar_wait_bounded(&full[i % slots], (i / slots) & 1u, &abort_flag))) {
            abort_flag = 1;
            if (lane == 0) atomicOr(a.error_word, kErrMbarTimeout);
        }
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            uint8_t *stage = tile + (i % slots) * stage_bytes;
            const uint32_t row = pos % kPageTokens;
            if (lo + i + 1u == pages && (row & ~15u) == key0) {  // this warp's keys include the token's own
                const uint4 *src = reinterpret_cast<const uint4 *>(new_row);
                for (uint32_t c = lane; c < (kb + VB) * 8u; c += 32u)
                    *reinterpret_cast<uint4 *>(stage + (c >> 3) * kBox + row * 128u + (((c & 7u) ^ (row & 7u)) << 4)) = src[c];
                __syncwarp();
            }
            const uint32_t base = smem_u32(stage);
            float sc[2][4] = {}, low[2][4] = {};  // products with the queries' leading and trailing halves
            const uint32_t key = key0 + (mi >> 1) * 8u + mr, key_line = base + key * 128u;
            for (uint32_t b = 0; b < kb; ++b) {
#pragma unroll
                for (uint32_t k16 = 0; k16 < 4u; ++k16) {  // 16 columns
                    uint32_t qh[4], ql[4], kf[4];
                    ldm(qh, q_at + (b * 64u + k16 * 16u) * 2u);
                    ldm(ql, q_lo_at + (b * 64u + k16 * 16u) * 2u);
                    ldm(kf, key_line + b * kBox + (((k16 * 2u + (mi & 1u)) ^ (key & 7u)) << 4));
                    mma_m16n8k16_bf16(sc[0], qh[0], qh[1], qh[2], qh[3], kf[0], kf[1]);
                    mma_m16n8k16_bf16(sc[1], qh[0], qh[1], qh[2], qh[3], kf[2], kf[3]);
                    mma_m16n8k16_bf16(low[0], ql[0], ql[1], ql[2], ql[3], kf[0], kf[1]);
                    mma_m16n8k16_bf16(low[1], ql[0], ql[1], ql[2], ql[3], kf[2], kf[3]);
                }
            }
            const uint32_t first_key = (lo + i) * kPageTokens + key0 + (lane & 3u) * 2u;
            if (first_key - (lane & 3u) * 2u <= pos) {  // the same for the whole warp
                float keep[2];
                uint32_t ph[4], pl[4];
#pragma unroll
                for (uint32_t r = 0; r < 2u; ++r) {  // rows lane / 4 and lane / 4 + 8
                    float v[4] = {sc[0][2u * r] + low[0][2u * r], sc[0][2u * r + 1u] + low[0][2u * r + 1u],
                                  sc[1][2u * r] + low[1][2u * r], sc[1][2u * r + 1u] + low[1][2u * r + 1u]};
                    float top = -INFINITY;
#pragma unroll
                    for (uint32_t e = 0; e < 4u; ++e) {
                        if (first_key + (e & 1u) + (e >> 1) * 8u > pos) v[e] = -INFINITY;
                        top = fmaxf(top, v[e]);
                    }
                    top = fmaxf(m[r], quad_max(top));
                    keep[r] = exp2f(m[r] - top);  // 0 at first
                    m[r] = top;
                    float sum = 0.0f;
#pragma unroll
                    for (uint32_t e = 0; e < 4u; ++e) {
                        v[e] = exp2f(v[e] - top);
                        sum += v[e];
                    }
                    l[r] = l[r] * keep[r] + quad_sum(sum);
                    split_bf16x2(v[0], v[1], ph[r], pl[r]);
                    split_bf16x2(v[2], v[3], ph[2u + r], pl[2u + r]);
                }
                const uint32_t vkey = key0 + (mi & 1u) * 8u + mr, value_line = base + kb * kBox + vkey * 128u;
#pragma unroll
                for (uint32_t b = 0; b < VB; ++b)
#pragma unroll
                    for (uint32_t n2 = 0; n2 < 4u; ++n2) {  // 16 columns
                        uint32_t vf[4];
                        ldm_trans(vf, value_line + b * kBox + (((n2 * 2u + (mi >> 1)) ^ (vkey & 7u)) << 4));
#pragma unroll
                        for (uint32_t t = 0; t < 2u; ++t) {
                            float(&o)[4] = out[b * 8u + n2 * 2u + t];
                            o[0] *= keep[0], o[1] *= keep[0], o[2] *= keep[1], o[3] *= keep[1];
                            mma_m16n8k16_bf16(o, ph[0], ph[1], ph[2], ph[3], vf[2u * t], vf[2u * t + 1u]);
                            mma_m16n8k16_bf16(o, pl[0], pl[1], pl[2], pl[3], vf[2u * t], vf[2u * t + 1u]);
                        }
                    }
            }
        }
        if (i0 + slots < n) {  // the two pages just read make room for two more
            __syncthreads();
            if (tid == 0)
                for (uint32_t j = i0 + slots; j < min(n, i0 + slots + 2u); ++j) fetch(j);
        }
    }

    // ---- merge of the warps: statistics, then weighted values, rows pitch apart
    const uint32_t pitch = s.vdim_p + 8u;
    float *state = reinterpret_cast<float *>(tile);  // [warp][head][pitch]; the sum ends up in warp 0's part
    if ((lane & 3u) == 0u) {
#pragma unroll
        for (uint32_t r = 0; r < 2u; ++r) warp_m[warp][(lane >> 2) + 8u * r] = m[r], warp_l[warp][(lane >> 2) + 8u * r] = l[r];
    }
    __syncthreads();  // everybody is through with the tiles as well
#pragma unroll
    for (uint32_t r = 0; r < 2u; ++r) {
        const uint32_t h = (lane >> 2) + 8u * r;
        if (h >= heads) continue;
        float top = -INFINITY, sum = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < kWarps; ++w) top = fmaxf(top, warp_m[w][h]);
        const float mine = m[r] == -INFINITY ? 0.0f : exp2f(m[r] - top);
        float *dst = state + ((size_t)warp * heads + h) * pitch + (lane & 3u) * 2u;
#pragma unroll
        for (uint32_t i = 0; i < VB * 8u; ++i)
            *reinterpret_cast<float2 *>(dst + i * 8u) = make_float2(out[i][2u * r] * mine, out[i][2u * r + 1u] * mine);
        if (warp == 0u && (lane & 3u) == 0u) {
#pragma unroll
            for (uint32_t w = 0; w < kWarps; ++w)
                if (warp_m[w][h] != -INFINITY) sum = fmaf(exp2f(warp_m[w][h] - top), warp_l[w][h], sum);
            run_m[h] = top, run_l[h] = sum;
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
        float weight[kMaxCluster], top = -INFINITY, sum = 0.0f;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (uint32_t c = 0; c < kMaxCluster; ++c) {
            weight[c] = c < a.cluster ? peer_load(peer_smem(&run_m[h], c)) : -INFINITY;
            top = fmaxf(top, weight[c]);
        }
#pragma unroll
        for (uint32_t c = 0; c < kMaxCluster; ++c) {
            if (c >= a.cluster) break;
            const float k = weight[c] == -INFINITY ? 0.0f : exp2f(weight[c] - top);
            sum = fmaf(k, peer_load(peer_smem(&run_l[h], c)), sum);
            const float4 x = peer_load4(peer_smem(state + h * pitch + q * 4u, c));
            v.x = fmaf(k, x.x, v.x), v.y = fmaf(k, x.y, v.y), v.z = fmaf(k, x.z, v.z), v.w = fmaf(k, x.w, v.w);
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
    if (a.cluster > 1u) cluster_sync();  // nobody leaves while another CTA may read its shared memory
}

struct Layout {
    uint32_t slots, tile_bytes, smem;
};
Layout layout_of(const GroupedShape &s) {
    const uint32_t stage = (s.dim_p + s.vdim_p) / 64u * kBox, heads = std::min(kHeads, s.per());
    Layout l{};
    l.slots = std::min(kMaxSlots, std::max(2u, kTileBudget / stage));
    l.tile_bytes = std::max(l.slots * stage, kWarps * heads * (s.vdim_p + 8u) * 4u);
    l.tile_bytes = (l.tile_bytes + 127u) & ~127u;
    l.smem = l.tile_bytes + 2u * kHeads * (s.dim_p + 8u) * 2u + (s.dim_p + s.vdim_p) * 2u + 1024u;
    return l;
}

using Kernel = void (*)(const CUtensorMap, const CUtensorMap, const GroupedArgs, uint32_t, uint32_t);
Kernel kernel_of(uint32_t value_blocks) {
    return value_blocks == 1u ? grouped_attend_mma_kernel<1>
                              : (value_blocks == 2u ? grouped_attend_mma_kernel<2>
                                                    : (value_blocks == 3u ? grouped_attend_mma_kernel<3> : grouped_attend_mma_kernel<4>));
}

}  // namespace

bool grouped_attend_mma_supports(const GroupedShape &s) {
    return s.dim_p <= kMaxBlocks * 64u && s.vdim_p <= kMaxBlocks * 64u && layout_of(s).smem <= kSmemLimit && encode_tiled() != nullptr;
}

stark_b200_status grouped_attend_mma_launch(const GroupedArgs &a, cudaStream_t stream) {
    const GroupedShape &s = a.s;
    if (!grouped_shape_supported(s, a.conv.taps) || !grouped_attend_mma_supports(s)) return STARK_B200_UNSUPPORTED;
    if (!a.u || a.u_b16 || a.cache_f32 || !a.conv.w || !a.conv.recent || !a.conv.tails || !a.keys || !a.values || !a.block_table ||
        !a.state || a.m != 1u || !a.temp_every || (a.mix != kMixNone && !a.first_values) || a.cluster == 0 ||
        a.cluster > kMaxCluster || (a.cluster & (a.cluster - 1u)) || a.splits == 0 || a.splits > kMaxSplits ||
        (a.splits == 1u ? !a.out : !a.partials))
        return STARK_B200_INVALID_ARGUMENT;
    const Kernel kernel = kernel_of(s.vdim_p / 64u);
    static SmemOptIn once[kMaxBlocks];
    if (stark_b200_status st = ensure_dynamic_smem(kernel, (int)kSmemLimit, once[s.vdim_p / 64u - 1u])) return st;
    CUtensorMap k_map, v_map;
    auto make = [&](CUtensorMap *map, void *base, uint32_t columns) {
        const cuuint64_t dims[2] = {columns, (cuuint64_t)a.num_blocks * s.groups * kPageTokens}, strides[1] = {(cuuint64_t)columns * 2u};
        const cuuint32_t box[2] = {64u, kPageTokens}, elem[2] = {1u, 1u};
        return encode_tiled()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, base, dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) ==
               CUDA_SUCCESS;
    };
    if (!make(&k_map, a.keys, s.dim_p) || !make(&v_map, a.values, s.vdim_p)) return STARK_B200_DEVICE_FAILURE;
    const Layout l = layout_of(s);
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
