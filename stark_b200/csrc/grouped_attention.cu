// Grouped-query attention with short convolutions: what happens to projected rows before they attend, for any number of
// rows, and the state the convolutions keep.  A unit is one head of the queries, keys or values; a warp owns one unit of a
// few rows.  Everything is f32 between the projected values and what is stored.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kThreads = 256, kWarpRows = 4, kCtaRows = kThreads / 32u * kWarpRows;
constexpr uint32_t kMaxBlocks = 8;  // heads up to 512 wide
constexpr uint32_t kWindowTaps = 4, kRun = 8;  // grouped_window_kernel: taps; rows in a run

// What a unit's channels are called in the projected row, and where its row goes.
struct Unit {
    bool is_q, is_k;
    uint32_t head, padded, blocks, col;
};
__device__ inline Unit unit_of(const GroupedShape &s, uint32_t unit, uint32_t lane) {
    Unit t;
    t.is_q = unit < s.heads, t.is_k = !t.is_q && unit < s.heads + s.groups;
    t.head = t.is_q ? unit : (t.is_k ? unit - s.heads : unit - s.heads - s.groups);
    t.padded = t.is_q || t.is_k ? s.dim_p : s.vdim_p;
    t.blocks = t.padded / 64u;
    t.col = (t.is_q ? 0u : (t.is_k ? s.key_col() : s.value_col())) + t.head * t.padded + lane * 2u;
    return t;
}

// Factor on a row of a query or key unit behind its convolution: norm, temperature, the scores' scale.
__device__ inline float row_factor(const GroupedArgs &a, const Unit &t, float sum_of_squares, uint32_t pos) {
    float factor = inverse_rms(sum_of_squares, a.s.dim, a.eps);
    if (t.is_q) {
        factor *= query_temperature(pos, a.temp_coef, a.temp_every);
        if (!a.queries_b16) factor *= a.scale * kLog2e;
    }
    return factor;
}

// One row of a unit to the queries or the cache, values mixed on the way.
template <typename E, uint32_t BLOCKS>
__device__ inline void store_row(const GroupedArgs &a, const Unit &t, uint32_t row, uint32_t pos, uint32_t page, uint32_t lane,
                                 const float2 (&v)[BLOCKS], float factor) {
    const GroupedShape &s = a.s;
    if (t.is_q) {
        const size_t at = ((size_t)row * s.heads + t.head) * s.dim_p + lane * 2u;
#pragma unroll
        for (uint32_t b = 0; b < BLOCKS; ++b) {
            if (b >= t.blocks) break;
            const float2 o = make_float2(v[b].x * factor, v[b].y * factor);
            if (a.queries_b16) store_pair(a.queries_b16 + at + b * 64u, o);
            else store_pair(a.queries + at + b * 64u, o);
        }
        return;
    }
    E *dst = reinterpret_cast<E *>(t.is_k ? a.keys : a.values) +
             (((size_t)page * s.groups + t.head) * kPageTokens + pos % kPageTokens) * t.padded + lane * 2u;
    float *first = a.first_values + ((size_t)row * s.groups + t.head) * s.vdim;  // values only
#pragma unroll
    for (uint32_t b = 0; b < BLOCKS; ++b) {
        if (b >= t.blocks) break;
        float2 o = make_float2(v[b].x * factor, v[b].y * factor);
        if (!t.is_k && a.mix == kMixFirst) keep_first_values(first, lane * 2u + b * 64u, s.vdim, o);
        if (!t.is_k && a.mix == kMixShare) o = mix_values(first, lane * 2u + b * 64u, s.vdim, o, a.share);
        store_pair(dst + b * 64u, o);
    }
}

// The projected row itself, where a later position's convolution will look for it.
template <typename E, uint32_t BLOCKS>
__device__ inline void keep_row(const GroupedArgs &a, const Unit &t, uint32_t pos, uint32_t page, const float2 (&x)[BLOCKS]) {
    const uint32_t taps = a.conv.taps, width = a.s.width(), in_page = pos % kPageTokens;
    const bool tail = in_page + taps > kPageTokens;  // one of the page's last taps - 1 positions
    E *recent = reinterpret_cast<E *>(a.conv.recent) + t.col, *tails = reinterpret_cast<E *>(a.conv.tails) + t.col;
#pragma unroll
    for (uint32_t b = 0; b < BLOCKS; ++b) {
        if (b >= t.blocks) break;
        if (a.m <= kConvSpare) store_pair(recent + (size_t)(pos % a.conv.recent_rows()) * width + b * 64u, x[b]);
        if (tail) store_pair(tails + ((size_t)page * (taps - 1u) + in_page + taps - 1u - kPageTokens) * width + b * 64u, x[b]);
    }
}

__device__ inline void unpack8(const uint4 &r, float (&v)[8]) {
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(w[i] << 16), v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
}

// Runs of kRun rows of a bf16 pass, up to kWindowTaps taps and heads up to 256 wide: what prompts go through.  A lane has
// eight neighbouring channels, as many lanes as the unit needs walk one run (a warp two or four runs of narrow units), the
// rows the convolution reaches stay in registers and every projected value is read once.  blockIdx: (rows, unit)
__global__ void __launch_bounds__(kThreads) grouped_window_kernel(const GroupedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const GroupedShape &s = a.s;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, taps = a.conv.taps, width = s.width();
    Unit t = unit_of(s, blockIdx.y, 0u);
    const uint32_t lanes = t.padded / 8u, runs = 32u / lanes, sub = lane / lanes, channel = lane % lanes * 8u;
    const bool idle = sub >= runs;  // 192 wide: eight lanes over
    const uint32_t warp_row0 = (blockIdx.x * (kThreads / 32u) + warp) * runs * kRun, row0 = warp_row0 + sub * kRun;
    if (warp_row0 >= a.m) return;
    t.col += channel;
    const uint16_t *u = reinterpret_cast<const uint16_t *>(a.u) + t.col;
    uint16_t *recent = reinterpret_cast<uint16_t *>(a.conv.recent) + t.col, *tails = reinterpret_cast<uint16_t *>(a.conv.tails) + t.col;
    const uint32_t rows = idle || row0 >= a.m ? 0u : min(kRun, a.m - row0);
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    uint4 raw[kRun], front[kWindowTaps - 1u];
#pragma unroll
    for (uint32_t r = 0; r < kRun; ++r)
        raw[r] = r < rows ? *reinterpret_cast<const uint4 *>(u + (size_t)(row0 + r) * a.ld_u) : zero;
    // the rows in front of the run: of this pass, or recent ones, or nothing (zeros) in front of the first token
#pragma unroll
    for (uint32_t i = 0; i < kWindowTaps - 1u; ++i) {
        const uint32_t back = kWindowTaps - 1u - i;
        front[i] = zero;
        if (rows && back < taps && back <= a.first_pos + row0)
            front[i] = *reinterpret_cast<const uint4 *>(
                back <= row0 ? u + (size_t)(row0 - back) * a.ld_u
                             : recent + (size_t)((a.first_pos + row0 - back) % a.conv.recent_rows()) * width);
    }
    float f[kWindowTaps][8];  // f[j] weighs the row kWindowTaps - 1 - j back
#pragma unroll
    for (uint32_t j = 0; j < kWindowTaps; ++j) {
        const bool in = !idle && j + taps >= kWindowTaps;
        const float4 *w = reinterpret_cast<const float4 *>(a.conv.w + (size_t)(in ? j + taps - kWindowTaps : 0u) * width + t.col);
        const float4 lo = in ? w[0] : make_float4(0.f, 0.f, 0.f, 0.f), hi = in ? w[1] : make_float4(0.f, 0.f, 0.f, 0.f);
        f[j][0] = lo.x, f[j][1] = lo.y, f[j][2] = lo.z, f[j][3] = lo.w, f[j][4] = hi.x, f[j][5] = hi.y, f[j][6] = hi.z, f[j][7] = hi.w;
    }
    // lane i: the page of the warp's row i, and its factor apart from the norm
    const uint32_t my_row = warp_row0 + lane, my_pos = a.first_pos + my_row;
    const bool mine = lane < runs * kRun && my_row < a.m;
    const uint32_t my_page = mine ? (uint32_t)a.block_table[my_pos / kPageTokens] : 0u;
    const float my_factor = t.is_q ? query_temperature(my_pos, a.temp_coef, a.temp_every) * (a.queries_b16 ? 1.0f : a.scale * kLog2e) : 1.0f;
    const float inverse_dim = 1.0f / (float)s.dim;
    float x[kWindowTaps][8];  // the window, by row modulo kWindowTaps
#pragma unroll
    for (uint32_t i = 0; i < kWindowTaps - 1u; ++i) unpack8(front[i], x[i]);
#pragma unroll
    for (uint32_t r = 0; r < kRun; ++r) {
        const uint32_t row = row0 + r, pos = a.first_pos + row;
        unpack8(raw[r], x[(r + kWindowTaps - 1u) % kWindowTaps]);
        float v[8], sum = 0.0f;
#pragma unroll
        for (uint32_t e = 0; e < 8u; ++e) {
            v[e] = 0.0f;
#pragma unroll
            for (uint32_t j = 0; j < kWindowTaps; ++j) v[e] = fmaf(f[j][e], x[(r + j) % kWindowTaps][e], v[e]);
            sum = fmaf(v[e], v[e], sum);
        }
        const uint32_t page = __shfl_sync(0xffffffffu, my_page, sub * kRun + r);
        if (t.is_q || t.is_k) {
            // over the run's lanes; all of the warp where they are no power of two (the idle ones hold zeros)
            for (uint32_t o = lanes == 24u ? 16u : lanes / 2u; o > 0u; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            const float factor = __shfl_sync(0xffffffffu, my_factor, sub * kRun + r) * rsqrtf(sum * inverse_dim + a.eps);
#pragma unroll
            for (uint32_t e = 0; e < 8u; ++e) v[e] *= factor;
        }
        if (r >= rows) continue;
        uint16_t *dst;
        if (t.is_q) {
            dst = a.queries_b16 + ((size_t)row * s.heads + t.head) * s.dim_p + channel;
        } else {
            dst = reinterpret_cast<uint16_t *>(t.is_k ? a.keys : a.values) +
                  (((size_t)page * s.groups + t.head) * kPageTokens + pos % kPageTokens) * t.padded + channel;
            if (!t.is_k && a.mix != kMixNone) {
                float *first = a.first_values + ((size_t)row * s.groups + t.head) * s.vdim;
#pragma unroll
                for (uint32_t e = 0; e < 8u; e += 2u) {
                    if (a.mix == kMixFirst) {
                        keep_first_values(first, channel + e, s.vdim, make_float2(v[e], v[e + 1u]));
                    } else {
                        const float2 o = mix_values(first, channel + e, s.vdim, make_float2(v[e], v[e + 1u]), a.share);
                        v[e] = o.x, v[e + 1u] = o.y;
                    }
                }
            }
        }
        *reinterpret_cast<uint4 *>(dst) = make_uint4(f32x2_to_bf16x2(v[0], v[1]), f32x2_to_bf16x2(v[2], v[3]),
                                                     f32x2_to_bf16x2(v[4], v[5]), f32x2_to_bf16x2(v[6], v[7]));
        // the projected row itself, where a later position's convolution will look for it
        const uint32_t in_page = pos % kPageTokens;
        if (taps > 1u && a.m <= kConvSpare) *reinterpret_cast<uint4 *>(recent + (size_t)(pos % a.conv.recent_rows()) * width) = raw[r];
        if (taps > 1u && in_page + taps > kPageTokens)
            *reinterpret_cast<uint4 *>(tails + ((size_t)page * (taps - 1u) + in_page + taps - 1u - kPageTokens) * width) = raw[r];
    }
}

// Any number of taps, heads up to kMaxBlocks blocks.  blockIdx: (rows, unit)
template <typename U, typename E>
__global__ void __launch_bounds__(kThreads) grouped_rows_kernel(const GroupedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, taps = a.conv.taps, width = a.s.width();
    const Unit t = unit_of(a.s, blockIdx.y, lane);
    const U *u = reinterpret_cast<const U *>(a.u) + t.col;
    const E *recent = reinterpret_cast<const E *>(a.conv.recent) + t.col;
    const float *w = a.conv.w + t.col;
    const uint32_t row0 = blockIdx.x * kCtaRows + warp * kWarpRows;
    for (uint32_t row = row0; row < min(a.m, row0 + kWarpRows); ++row) {
        const uint32_t pos = a.state ? a.state->position : a.first_pos + row, page = (uint32_t)a.block_table[pos / kPageTokens];
        float2 v[kMaxBlocks], x[kMaxBlocks];
        float sum = 0.0f;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            if (b >= t.blocks) break;
            float2 acc = make_float2(0.0f, 0.0f);
            for (uint32_t j = 0; j < taps; ++j) {
                const uint32_t back = taps - 1u - j;
                if (back > pos) continue;  // nothing precedes the first token
                x[b] = back <= row ? load_pair(u + (size_t)(row - back) * a.ld_u + b * 64u)
                                   : load_pair(recent + (size_t)((pos - back) % a.conv.recent_rows()) * width + b * 64u);
                const float2 f = load_pair(w + (size_t)j * width + b * 64u);
                acc.x = fmaf(f.x, x[b].x, acc.x), acc.y = fmaf(f.y, x[b].y, acc.y);
            }
            v[b] = acc;
            sum += acc.x * acc.x + acc.y * acc.y;
        }
        const float factor = t.is_q || t.is_k ? row_factor(a, t, warp_sum(sum), pos) : 1.0f;
        store_row<E, kMaxBlocks>(a, t, row, pos, page, lane, v, factor);
        if (taps > 1u) keep_row<E, kMaxBlocks>(a, t, pos, page, x);  // the last x is the row's own
    }
}

// The last taps - 1 rows of a pass into the recent rows.  One CTA per row.
template <typename U, typename E>
__global__ void __launch_bounds__(kThreads) short_conv_keep_kernel(const GroupedArgs a) {
    const uint32_t width = a.s.width(), row = a.m - 1u - blockIdx.x;
    const U *src = reinterpret_cast<const U *>(a.u) + (size_t)row * a.ld_u;
    E *dst = reinterpret_cast<E *>(a.conv.recent) + (size_t)((a.first_pos + row) % a.conv.recent_rows()) * width;
    for (uint32_t i = threadIdx.x * 2u; i < width; i += kThreads * 2u) store_pair(dst + i, load_pair(src + i));
}

template <typename E>
__global__ void __launch_bounds__(kThreads) short_conv_restore_kernel(const GroupedArgs a, uint32_t position) {
    const uint32_t width = a.s.width(), pos = position - 1u - blockIdx.x, page = (uint32_t)a.block_table[pos / kPageTokens];
    const uint32_t in_tail = pos % kPageTokens + a.conv.taps - 1u - kPageTokens;
    const E *src = reinterpret_cast<const E *>(a.conv.tails) + ((size_t)page * (a.conv.taps - 1u) + in_tail) * width;
    E *dst = reinterpret_cast<E *>(a.conv.recent) + (size_t)(pos % a.conv.recent_rows()) * width;
    for (uint32_t i = threadIdx.x; i < width; i += kThreads) dst[i] = src[i];
}

}  // namespace

bool grouped_shape_supported(const GroupedShape &s, uint32_t taps) {
    return s.heads && s.groups && s.heads % s.groups == 0 && s.dim && s.vdim && s.dim_p <= kMaxBlocks * 64u &&
           s.vdim_p <= kMaxBlocks * 64u && taps >= 1u && taps <= kPageTokens && s.heads + 2u * s.groups <= 65535u;
}

stark_b200_status grouped_rows_launch(const GroupedArgs &a, cudaStream_t stream) {
    if (!grouped_shape_supported(a.s, a.conv.taps)) return STARK_B200_UNSUPPORTED;
    if (!a.u || !a.conv.w || !a.conv.recent || !a.conv.tails || !a.keys || !a.values || !a.block_table || a.m == 0 ||
        (a.state && a.m != 1u) || !a.temp_every || (a.mix != kMixNone && !a.first_values) ||
        (a.queries == nullptr) == (a.queries_b16 == nullptr) || (a.u_b16 && a.cache_f32) || a.ld_u < a.s.width() || a.ld_u % 2u)
        return STARK_B200_INVALID_ARGUMENT;
    const uint32_t units = a.s.heads + 2u * a.s.groups, widest = std::max(a.s.dim_p, a.s.vdim_p);
    if (a.u_b16 && a.queries_b16 && a.conv.taps <= kWindowTaps && widest <= 256u && a.ld_u % 8u == 0) {
        const uint32_t cta_rows = kThreads / 32u * (256u / widest) * kRun;  // of the units with the fewest runs to a warp
        if (stark_b200_status st = launch_chained(grouped_window_kernel, dim3((a.m + cta_rows - 1u) / cta_rows, units), dim3(kThreads), 0,
                                                  a.pdl, stream, a))
            return st;
    } else {
        auto kernel = a.u_b16 ? grouped_rows_kernel<uint16_t, uint16_t>
                              : (a.cache_f32 ? grouped_rows_kernel<float, float> : grouped_rows_kernel<float, uint16_t>);
        if (stark_b200_status st = launch_chained(kernel, dim3((a.m + kCtaRows - 1u) / kCtaRows, units), dim3(kThreads), 0, a.pdl, stream, a))
            return st;
    }
    if (a.m <= kConvSpare || a.conv.taps == 1u) return STARK_B200_OK;
    auto keep = a.u_b16 ? short_conv_keep_kernel<uint16_t, uint16_t>
                        : (a.cache_f32 ? short_conv_keep_kernel<float, float> : short_conv_keep_kernel<float, uint16_t>);
    keep<<<std::min(a.m, a.conv.taps - 1u), kThreads, 0, stream>>>(a);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

stark_b200_status short_conv_restore_launch(const GroupedArgs &a, uint32_t position, cudaStream_t stream) {
    if (position % kPageTokens || !a.conv.recent || !a.conv.tails) return STARK_B200_INVALID_ARGUMENT;
    if (position == 0 || a.conv.taps == 1u) return STARK_B200_OK;
    auto kernel = a.cache_f32 ? short_conv_restore_kernel<float> : short_conv_restore_kernel<uint16_t>;
    kernel<<<a.conv.taps - 1u, kThreads, 0, stream>>>(a, position);
    SB_CUDA(cudaGetLastError());
    return STARK_B200_OK;
}

}  // namespace sb
