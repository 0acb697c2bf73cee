// Grouped-query attention with short convolutions: what happens to projected rows before they attend, for any number of
// rows, and the state the convolutions keep.  A unit is one head of the queries, keys or values; a warp owns one unit of a
// few rows, two neighbouring channels a lane and 64 channels at a time.  Everything is f32 between the projected values and
// what is stored.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kThreads = 256, kWarpRows = 8, kCtaRows = kThreads / 32u * kWarpRows;
constexpr uint32_t kMaxBlocks = 8;  // heads up to 512 wide
constexpr uint32_t kWindowTaps = 4, kWindowBlocks = 2;

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

// Sums over the warp's lanes of eight values each, by halves: afterwards lane l holds the sum of value (l >> 2) with its
// three bits in reverse, which is row_of_lane(l).
__device__ inline uint32_t row_of_lane(uint32_t lane) { return ((lane >> 4) & 1u) | ((lane >> 2) & 2u) | (lane & 4u); }
__device__ inline uint32_t lane_of_row(uint32_t row) { return ((row & 1u) << 4) | ((row & 2u) << 2) | (row & 4u); }
__device__ inline float sum_eight(const float (&v)[8], uint32_t lane) {
    float a[4], b[2], c;
#pragma unroll
    for (uint32_t i = 0; i < 4u; ++i) {
        const bool up = (lane & 16u) != 0u;
        const float send = up ? v[2u * i] : v[2u * i + 1u], keep = up ? v[2u * i + 1u] : v[2u * i];
        a[i] = keep + __shfl_xor_sync(0xffffffffu, send, 16);
    }
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
        const bool up = (lane & 8u) != 0u;
        const float send = up ? a[2u * i] : a[2u * i + 1u], keep = up ? a[2u * i + 1u] : a[2u * i];
        b[i] = keep + __shfl_xor_sync(0xffffffffu, send, 8);
    }
    const bool up = (lane & 4u) != 0u;
    c = (up ? b[1] : b[0]) + __shfl_xor_sync(0xffffffffu, up ? b[0] : b[1], 4);
    c += __shfl_xor_sync(0xffffffffu, c, 2);
    return c + __shfl_xor_sync(0xffffffffu, c, 1);
}

// Up to kWindowTaps taps and heads of kWindowBlocks blocks: a warp holds the rows its convolution reaches in registers, all
// of them asked for at once, so that a projected value is read once (and the few rows in front of a warp's first one again);
// the norms of its eight rows are reduced together and each row's factor is worked out by the lanes that end up with it.
// U: type of the projected rows; E: type of the cache and of the convolutions' state.  blockIdx: (rows, unit)
template <typename U, typename E>
__global__ void __launch_bounds__(kThreads) grouped_window_kernel(const GroupedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    using RawU = RawPair<U>;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, taps = a.conv.taps, width = a.s.width();
    const Unit t = unit_of(a.s, blockIdx.y, lane);
    const uint32_t row0 = blockIdx.x * kCtaRows + warp * kWarpRows;
    if (row0 >= a.m) return;
    const uint32_t first_pos = a.state ? a.state->position : a.first_pos, rows = min(kWarpRows, a.m - row0);
    const U *u = reinterpret_cast<const U *>(a.u) + (size_t)row0 * a.ld_u + t.col;
    constexpr uint32_t kBack = kWindowTaps - 1u;
    typename RawU::type x[kBack + kWarpRows][kWindowBlocks];
    float2 f[kWindowTaps][kWindowBlocks];  // f[j] weighs the row kBack - j back
#pragma unroll
    for (uint32_t i = 0; i < kWarpRows; ++i)
#pragma unroll
        for (uint32_t b = 0; b < kWindowBlocks; ++b)
            x[kBack + i][b] = i < rows && b < t.blocks
                                  ? *reinterpret_cast<const typename RawU::type *>(u + (size_t)i * a.ld_u + b * 64u)
                                  : RawU::zero();
    // the rows in front: of this pass, or recent ones, or zeros before the sequence's start
    float2 front[kBack][kWindowBlocks];
#pragma unroll
    for (uint32_t i = 0; i < kBack; ++i) {
        const uint32_t back = kBack - i;
        const bool in = back < taps && back <= first_pos + row0;
        const E *recent = reinterpret_cast<const E *>(a.conv.recent) + (size_t)((first_pos + row0 - (in ? back : 0u)) % a.conv.recent_rows()) * width + t.col;
#pragma unroll
        for (uint32_t b = 0; b < kWindowBlocks; ++b) {
            front[i][b] = make_float2(0.0f, 0.0f);
            if (in && b < t.blocks) front[i][b] = back <= row0 ? load_pair(u - (size_t)back * a.ld_u + b * 64u) : load_pair(recent + b * 64u);
        }
    }
#pragma unroll
    for (uint32_t j = 0; j < kWindowTaps; ++j)
#pragma unroll
        for (uint32_t b = 0; b < kWindowBlocks; ++b)
            f[j][b] = j + taps >= kWindowTaps && b < t.blocks ? load_pair(a.conv.w + (size_t)(j + taps - kWindowTaps) * width + t.col + b * 64u)
                                                              : make_float2(0.0f, 0.0f);
    // lane r < kWarpRows: the page of row r
    const uint32_t my_page = lane < rows ? (uint32_t)a.block_table[(first_pos + row0 + lane) / kPageTokens] : 0u;
    float2 v[kWarpRows][kWindowBlocks];
    float squares[kWarpRows];
#pragma unroll
    for (uint32_t r = 0; r < kWarpRows; ++r) {
        squares[r] = 0.0f;
#pragma unroll
        for (uint32_t b = 0; b < kWindowBlocks; ++b) {
            float2 acc = make_float2(0.0f, 0.0f);
#pragma unroll
            for (uint32_t j = 0; j < kWindowTaps; ++j) {
                const float2 at = r + j < kBack ? front[r + j][b] : RawU::value(x[r + j][b]);
                acc.x = fmaf(f[j][b].x, at.x, acc.x), acc.y = fmaf(f[j][b].y, at.y, acc.y);
            }
            v[r][b] = acc;
            squares[r] += acc.x * acc.x + acc.y * acc.y;
        }
    }
    float my_factor = 1.0f;
    if (t.is_q || t.is_k) my_factor = row_factor(a, t, sum_eight(squares, lane), first_pos + row0 + row_of_lane(lane));
#pragma unroll
    for (uint32_t r = 0; r < kWarpRows; ++r) {
        if (r >= rows) break;
        const uint32_t pos = first_pos + row0 + r, page = __shfl_sync(0xffffffffu, my_page, r);
        const float factor = __shfl_sync(0xffffffffu, my_factor, lane_of_row(r));
        store_row<E, kWindowBlocks>(a, t, row0 + r, pos, page, lane, v[r], factor);
        if (taps > 1u && (a.m <= kConvSpare || pos % kPageTokens + taps > kPageTokens)) {
            float2 raw[kWindowBlocks];
#pragma unroll
            for (uint32_t b = 0; b < kWindowBlocks; ++b) raw[b] = RawU::value(x[r + kBack][b]);
            keep_row<E, kWindowBlocks>(a, t, pos, page, raw);
        }
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
                if (back > pos) continue;  // zeros before the sequence's start
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
    const bool window = a.conv.taps <= kWindowTaps && std::max(a.s.dim_p, a.s.vdim_p) <= kWindowBlocks * 64u;
    auto kernel = window ? (a.u_b16 ? grouped_window_kernel<uint16_t, uint16_t>
                                    : (a.cache_f32 ? grouped_window_kernel<float, float> : grouped_window_kernel<float, uint16_t>))
                         : (a.u_b16 ? grouped_rows_kernel<uint16_t, uint16_t>
                                    : (a.cache_f32 ? grouped_rows_kernel<float, float> : grouped_rows_kernel<float, uint16_t>));
    const dim3 grid((a.m + kCtaRows - 1u) / kCtaRows, a.s.heads + 2u * a.s.groups);
    if (stark_b200_status st = launch_chained(kernel, grid, dim3(kThreads), 0, a.pdl, stream, a)) return st;
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
