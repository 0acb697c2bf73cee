// Grouped-query attention with short convolutions: what happens to projected rows before they attend, for any number of
// rows, and the state the convolutions keep.  A unit is one head of the queries, keys or values; a warp owns one unit of a
// few rows, two neighbouring channels a lane and 64 channels at a time.  Everything is f32 between the projected values and
// what is stored.
#include "layered.cuh"
#include "layered_math.cuh"

namespace sb {

namespace {

constexpr uint32_t kThreads = 256, kWarpRows = 4, kCtaRows = kThreads / 32u * kWarpRows;
constexpr uint32_t kMaxBlocks = 8;  // heads up to 512 wide

// U: type of the projected rows; E: type of the cache and of the convolutions' state.  blockIdx: (rows, unit)
template <typename U, typename E>
__global__ void __launch_bounds__(kThreads) grouped_rows_kernel(const GroupedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const GroupedShape &s = a.s;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, unit = blockIdx.y;
    const bool is_q = unit < s.heads, is_k = !is_q && unit < s.heads + s.groups;
    const uint32_t head = is_q ? unit : (is_k ? unit - s.heads : unit - s.heads - s.groups);
    const uint32_t padded = is_q || is_k ? s.dim_p : s.vdim_p, blocks = padded / 64u;
    const uint32_t col = (is_q ? 0u : (is_k ? s.key_col() : s.value_col())) + head * padded + lane * 2u;
    const uint32_t width = s.width(), taps = a.conv.taps, recent_rows = a.conv.recent_rows();
    const U *u = reinterpret_cast<const U *>(a.u) + col;
    E *recent = reinterpret_cast<E *>(a.conv.recent) + col, *tails = reinterpret_cast<E *>(a.conv.tails) + col;
    const float *w = a.conv.w + col;
    const uint32_t row0 = blockIdx.x * kCtaRows + warp * kWarpRows;
    for (uint32_t row = row0; row < min(a.m, row0 + kWarpRows); ++row) {
        const uint32_t pos = a.state ? a.state->position : a.first_pos + row;
        float2 v[kMaxBlocks];
        float sum = 0.0f;
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            if (b >= blocks) break;
            float2 acc = make_float2(0.0f, 0.0f);
            for (uint32_t j = 0; j < taps; ++j) {
                const uint32_t back = taps - 1u - j;
                if (back > pos) continue;  // zeros before the sequence's start
                const float2 x = back <= row ? load_pair(u + (size_t)(row - back) * a.ld_u + b * 64u)
                                             : load_pair(recent + (size_t)((pos - back) % recent_rows) * width + b * 64u);
                const float2 f = load_pair(w + (size_t)j * width + b * 64u);
                acc.x = fmaf(f.x, x.x, acc.x), acc.y = fmaf(f.y, x.y, acc.y);
            }
            v[b] = acc;
            sum += acc.x * acc.x + acc.y * acc.y;
        }
        const uint32_t page = (uint32_t)a.block_table[pos / kPageTokens], in_page = pos % kPageTokens;
        float factor = 1.0f;
        if (is_q || is_k) {
            factor = inverse_rms(warp_sum(sum), s.dim, a.eps);
            if (is_q) {
                factor *= query_temperature(pos, a.temp_coef, a.temp_every);
                if (!a.queries_b16) factor *= a.scale * kLog2e;
            }
        }
        E *dst = reinterpret_cast<E *>(is_k ? a.keys : a.values) +
                 (((size_t)page * s.groups + head) * kPageTokens + in_page) * padded + lane * 2u;  // not used by queries
        float *first = a.first_values + (size_t)row * s.groups * s.vdim + head * s.vdim;  // values only
#pragma unroll
        for (uint32_t b = 0; b < kMaxBlocks; ++b) {
            if (b >= blocks) break;
            float2 o = make_float2(v[b].x * factor, v[b].y * factor);
            if (is_q) {
                const size_t at = ((size_t)row * s.heads + head) * s.dim_p + lane * 2u + b * 64u;
                if (a.queries_b16) store_pair(a.queries_b16 + at, o);
                else store_pair(a.queries + at, o);
            } else {
                if (!is_k && a.mix == kMixFirst) keep_first_values(first, lane * 2u + b * 64u, s.vdim, o);
                if (!is_k && a.mix == kMixShare) o = mix_values(first, lane * 2u + b * 64u, s.vdim, o, a.share);
                store_pair(dst + b * 64u, o);
            }
        }
        // the projected row itself, where a later position's convolution will look for it
        const bool tail = in_page + taps > kPageTokens;  // one of the page's last taps - 1 positions
        if (taps > 1u && (tail || a.m <= kConvSpare)) {
#pragma unroll
            for (uint32_t b = 0; b < kMaxBlocks; ++b) {
                if (b >= blocks) break;
                const float2 x = load_pair(u + (size_t)row * a.ld_u + b * 64u);
                if (a.m <= kConvSpare) store_pair(recent + (size_t)(pos % recent_rows) * width + b * 64u, x);
                if (tail) store_pair(tails + ((size_t)page * (taps - 1u) + in_page + taps - 1u - kPageTokens) * width + b * 64u, x);
            }
        }
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
    auto kernel = a.u_b16 ? grouped_rows_kernel<uint16_t, uint16_t>
                          : (a.cache_f32 ? grouped_rows_kernel<float, float> : grouped_rows_kernel<float, uint16_t>);
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
