// Row-wise operators of the bfloat16 decoders, all in fp32: embedding rows with learned positions, the end of a sublayer
// (grouped RMS norm of its output, residual add, token shift or output norm for whatever reads the stream next), per-head norms
// with a gate, and query/key norms or convolution and rotation with the KV append.
//
// The end of a sublayer is a device function, because it runs in two places: as a kernel over the rows of a block
// (sublayer_end_rows_kernel) and in the prologue of the decode product that consumes its result (gemv_bf16.cuh).
//
// Every kernel is launched with programmatic stream serialisation and waits for the previous grid before it touches memory.
#pragma once
#include <cuda_bf16.h>

#include <cstdint>

#include "attention.cuh"
#include "zk_ptx.cuh"

namespace zk {

// x_new = x_in + norm(y), or x_in alone without y_a; per row of n values.
//   y         = y_a, or with y_b half the sum of both after each is divided by its root mean square and multiplied by
//               weight_a / weight_b
//   norm      = groups equal consecutive parts, each divided by its own root mean square, times norm_weight; without norm_weight
//               the residual add is plain: x_new = x_in + y
// The row's consumer gets h = x_new + (before - x_new) * shift (before: the previous token's x_new), or the grouped norm of x_new
// with out_norm, or x_new itself.  keep receives the block's last row of x_in: the sublayer's own input, which the sequence's next
// token reads as `before`.
struct SublayerEnd {
    const float* x_in;
    float* x_out;             // null: x_new is not stored
    const float* y_a;
    const float* y_b;
    const float* weight_a;
    const float* weight_b;
    const float* norm_weight;
    float* keep;
    const float* shift;
    const float* before;      // [n]: the token before the block's first
    const float* out_norm;
    uint32_t n, groups;
    float eps;
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Floats of scratch the block-wide functions below need beside the row itself.
__host__ __device__ inline uint32_t row_scratch_floats(uint32_t threads, uint32_t groups) {
    const uint32_t warps = threads / 32;
    return (warps > groups ? warps : groups) + groups + 2 * warps;
}

// scratch[g] = 1 / sqrt(mean over part g of row^2 + eps), for every one of the block's threads; returns the table.
template <int kThreads>
__device__ __forceinline__ const float* group_inverse_rms(const float* row, uint32_t n, uint32_t groups, float eps, float* scratch) {
    constexpr uint32_t kWarps = kThreads / 32;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, size = n / groups;
    const uint32_t per = groups < kWarps ? kWarps / groups : 1u;        // warps per part
    float* sums = scratch;
    float* inverse = scratch + (kWarps > groups ? kWarps : groups);
    for (uint32_t u = warp; u < groups * per; u += kWarps) {
        const float* part = row + (u / per) * size;
        float s = 0.0f;
        for (uint32_t i = (u % per) * 32 + lane; i < size; i += per * 32) s += part[i] * part[i];
        s = warp_sum(s);
        if (lane == 0) sums[u] = s;
    }
    __syncthreads();
    for (uint32_t g = threadIdx.x; g < groups; g += kThreads) {
        float s = 0.0f;
        for (uint32_t j = 0; j < per; ++j) s += sums[g * per + j];
        inverse[g] = 1.0f / sqrtf(s / static_cast<float>(size) + eps);
    }
    __syncthreads();
    return inverse;
}

// x_new of one row into shared memory (row[n]); all threads of the block.  Ends with a barrier.
template <int kThreads>
__device__ __forceinline__ void sublayer_row(const SublayerEnd& p, size_t r, float* row, float* scratch) {
    const float* x = p.x_in + r * p.n;
    if (!p.y_a) {
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] = __ldcg(x + i);
        __syncthreads();
        return;
    }
    const float* a = p.y_a + r * p.n;
    if (!p.norm_weight) {
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] = __ldcg(x + i) + __ldcg(a + i);
        __syncthreads();
        return;
    }
    if (p.y_b) {
        constexpr uint32_t kWarps = kThreads / 32;
        const float* b = p.y_b + r * p.n;
        float sa = 0.0f, sb = 0.0f;
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) {
            const float va = __ldcg(a + i), vb = __ldcg(b + i);
            sa += va * va;
            sb += vb * vb;
        }
        sa = warp_sum(sa);
        sb = warp_sum(sb);
        float* part = scratch + row_scratch_floats(kThreads, p.groups) - 2 * kWarps;
        if ((threadIdx.x & 31) == 0) { part[threadIdx.x >> 5] = sa; part[kWarps + (threadIdx.x >> 5)] = sb; }
        __syncthreads();
        sa = sb = 0.0f;
        for (uint32_t w = 0; w < kWarps; ++w) { sa += part[w]; sb += part[kWarps + w]; }
        const float ra = 1.0f / sqrtf(sa / static_cast<float>(p.n) + p.eps), rb = 1.0f / sqrtf(sb / static_cast<float>(p.n) + p.eps);
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads)
            row[i] = 0.5f * (__ldcg(a + i) * ra * p.weight_a[i] + __ldcg(b + i) * rb * p.weight_b[i]);
    } else {
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] = __ldcg(a + i);
    }
    __syncthreads();
    const float* inverse = group_inverse_rms<kThreads>(row, p.n, p.groups, p.eps, scratch);
    const uint32_t size = p.n / p.groups;
    for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] = __ldcg(x + i) + row[i] * inverse[i / size] * p.norm_weight[i];
    __syncthreads();
}

// What the consumer reads, from x_new in shared memory, in place.  before_row: the previous token's x_new (only read with shift).
template <int kThreads>
__device__ __forceinline__ void sublayer_view(const SublayerEnd& p, float* row, const float* before_row, float* scratch) {
    if (p.shift) {
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] += (before_row[i] - row[i]) * p.shift[i];
    } else if (p.out_norm) {
        const float* inverse = group_inverse_rms<kThreads>(row, p.n, p.groups, p.eps, scratch);
        const uint32_t size = p.n / p.groups;
        for (uint32_t i = threadIdx.x; i < p.n; i += kThreads) row[i] = row[i] * inverse[i / size] * p.out_norm[i];
    }
    __syncthreads();
}

__device__ __forceinline__ void store_as(float* dst, float v) { *dst = v; }
__device__ __forceinline__ void store_as(__nv_bfloat16* dst, float v) { *dst = __float2bfloat16_rn(v); }

// The end of a sublayer over a block of rows, one CTA per row; view [rows][ld] (bf16 or fp32; columns n .. ld - 1 are written as
// zeros) is the next product's input, or null.  With a token shift a CTA computes the row before its own as well: x_in and x_out
// are different buffers, so it does not matter which CTA gets there first.
constexpr int kRowThreads = 256;
template <typename TView>
__global__ void __launch_bounds__(kRowThreads) sublayer_end_rows_kernel(const __grid_constant__ SublayerEnd p, TView* __restrict__ view, uint32_t ld) {
    extern __shared__ float row_smem[];
    float* row = row_smem;
    float* before = row_smem + p.n;                 // used only with a shift
    float* scratch = p.shift ? before + p.n : before;
    pdl_launch_dependents();
    pdl_wait();
    const size_t r = blockIdx.x;
    sublayer_row<kRowThreads>(p, r, row, scratch);
    if (p.x_out)
        for (uint32_t i = threadIdx.x; i < p.n; i += kRowThreads) p.x_out[r * p.n + i] = row[i];
    if (p.keep && r + 1 == gridDim.x)
        for (uint32_t i = threadIdx.x; i < p.n; i += kRowThreads) p.keep[i] = p.x_in[r * p.n + i];
    if (!view) return;
    if (p.shift) {
        if (r > 0) {
            sublayer_row<kRowThreads>(p, r - 1, before, scratch);
        } else {
            for (uint32_t i = threadIdx.x; i < p.n; i += kRowThreads) before[i] = p.before[i];
            __syncthreads();
        }
    }
    sublayer_view<kRowThreads>(p, row, before, scratch);
    for (uint32_t i = threadIdx.x; i < ld; i += kRowThreads) store_as(view + r * ld + i, i < p.n ? row[i] : 0.0f);
}

// out[t] = embed[tokens[t]] + positions[*pos + t] (positions null: the embedding alone); grid (ceil(n / 256), T).
__global__ void __launch_bounds__(256) embed_rows_bf16_kernel(const __nv_bfloat16* __restrict__ embed, uint32_t vocab, uint32_t ld,
                                                              const __nv_bfloat16* __restrict__ positions, uint32_t max_positions, uint32_t pos_ld,
                                                              const long long* __restrict__ tokens, const int* __restrict__ pos_ptr,
                                                              float* __restrict__ out, uint32_t n, int* error_word) {
    pdl_launch_dependents();
    pdl_wait();
    const long long id = tokens[blockIdx.y], pos = positions ? static_cast<long long>(*pos_ptr) + blockIdx.y : 0;
    const bool good_id = id >= 0 && id < static_cast<long long>(vocab), good_pos = !positions || (pos >= 0 && pos < static_cast<long long>(max_positions));
    if (threadIdx.x == 0 && blockIdx.x == 0) {
        if (!good_id) atomicExch(error_word, kErrBadToken);
        else if (!good_pos) atomicExch(error_word, kErrBadPosition);
    }
    const uint32_t i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    float v = 0.0f;
    if (good_id && good_pos) {
        v = __bfloat162float(embed[static_cast<size_t>(id) * ld + i]);
        if (positions) v += __bfloat162float(positions[static_cast<size_t>(pos) * pos_ld + i]);
    }
    out[static_cast<size_t>(blockIdx.y) * n + i] = v;
}

// Columns [0, n) of rows of pitch src_ld as the next product's input [rows][ld], zeros behind them.
template <typename TView>
__global__ void __launch_bounds__(256) rows_view_kernel(const float* __restrict__ src, uint32_t src_ld, uint32_t n, TView* __restrict__ dst, uint32_t ld) {
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t i = threadIdx.x; i < ld; i += 256)
        store_as(dst + static_cast<size_t>(blockIdx.x) * ld + i, i < n ? src[static_cast<size_t>(blockIdx.x) * src_ld + i] : 0.0f);
}

// Per head of `width` values (input pitch head_ld): o, divided by its root mean square and times weight when weight is given,
// times a gate.  gate_mode 0: none; 1: sigmoid, one value per head, gate [rows][gate_ld]; 2 and 3: sigmoid or silu, one per value,
// [rows][gate_ld], laid out heads x width.  dst [rows][ld] packs the heads without padding, zeros behind them up to column `fill`.
// A warp takes a head; grid: rows.
template <typename TView>
__global__ void __launch_bounds__(256) head_outputs_rows_kernel(const float* __restrict__ o, uint32_t heads, uint32_t width, uint32_t head_ld,
                                                                const float* __restrict__ weight, float eps, const float* __restrict__ gate, uint32_t gate_ld,
                                                                int gate_mode, TView* __restrict__ dst, uint32_t ld, uint32_t fill) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t r = blockIdx.x;
    for (uint32_t h = warp; h < heads; h += 8) {
        const float* v = o + (r * heads + h) * head_ld;
        float inv = 1.0f;
        if (weight) {
            float ss = 0.0f;
            for (uint32_t i = lane; i < width; i += 32) ss += v[i] * v[i];
            inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(width) + eps);
        }
        const float head_gate = gate_mode == 1 ? logistic(gate[r * gate_ld + h]) : 1.0f;
        for (uint32_t i = lane; i < width; i += 32) {
            float y = v[i] * inv * head_gate;
            if (weight) y *= weight[i];
            if (gate_mode >= 2) {
                const float z = gate[r * gate_ld + h * width + i];
                y *= gate_mode == 2 ? logistic(z) : silu_f(z);
            }
            store_as(dst + r * ld + h * width + i, y);
        }
    }
    for (uint32_t i = heads * width + threadIdx.x; i < fill; i += 256) store_as(dst + r * ld + i, 0.0f);
}

// Query and key norms of a block of rows and the append of its keys and values at positions *pos ..: q, k, v are columns of the
// projection rows (pitch ld); q_out [rows][heads][pitch] and the caches [positions][kv_heads][pitch] are zero beyond the real
// sizes.  A warp takes a head; grid: rows.
__global__ void __launch_bounds__(256) qk_norm_append_rows_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, uint32_t ld,
                                                                  AttnWindow win, uint32_t heads, uint32_t kv_heads, uint32_t pitch,
                                                                  const int* __restrict__ pos_ptr, float* __restrict__ q_out, float* __restrict__ k_cache,
                                                                  float* __restrict__ v_cache, uint32_t max_positions, int* error_word) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t r = blockIdx.x;
    const long long pos = static_cast<long long>(*pos_ptr) + blockIdx.x;
    if (pos < 0 || pos >= static_cast<long long>(max_positions)) {
        if (threadIdx.x == 0) atomicExch(error_word, kErrBadPosition);
        return;
    }
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (uint32_t h = warp; h < heads + 2 * kv_heads; h += 8) {
        const bool is_q = h < heads, is_k = !is_q && h < heads + kv_heads;
        const uint32_t g = is_q ? h : is_k ? h - heads : h - heads - kv_heads, n = is_q || is_k ? win.qk_dim : win.v_dim;
        const float* src = (is_q ? q : is_k ? k : v) + r * ld + g * n;
        float* dst = is_q ? q_out + (r * heads + g) * pitch : (is_k ? k_cache : v_cache) + (static_cast<size_t>(pos) * kv_heads + g) * pitch;
        float inv = 1.0f;
        if (is_q || is_k) {
            float ss = 0.0f;
            for (uint32_t i = lane; i < n; i += 32) ss += src[i] * src[i];
            inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(n) + win.eps);
        }
        const float* w = is_q ? win.q_weight : win.k_weight;
        for (uint32_t i = lane; i < pitch; i += 32) dst[i] = i < n ? ((is_q || is_k) ? src[i] * inv * w[i] : src[i]) : 0.0f;
    }
}

// The ring after a block of T tokens: the inputs of its last min(T, taps) tokens.  Runs after every reader of the ring; x: the
// channels' columns of the projection rows.
__global__ void __launch_bounds__(256) conv_ring_update_kernel(const __grid_constant__ ShortConv conv, const float* __restrict__ x, uint32_t ld, uint32_t tokens,
                                                               const int* __restrict__ pos_ptr) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t c = blockIdx.x * 256 + threadIdx.x, pos = static_cast<uint32_t>(*pos_ptr);
    if (c >= conv.channels) return;
    for (uint32_t t = tokens > conv.taps ? tokens - conv.taps : 0; t < tokens; ++t)
        conv.ring[static_cast<size_t>((pos + t) % conv.taps) * conv.channels + c] = x[static_cast<size_t>(t) * ld + c];
}

// The rotary form of the norm-and-append kernel: per channel of q, k and v the short convolution, then the rotation of q and k, the mixing of v
// with the values of an earlier layer (or their keeping for later layers), and the append.  A warp takes (strip of kStrip tokens,
// head); grid: (strips, CTAs that share one).  The ring is brought up to date afterwards (conv_ring_update_kernel).
__global__ void __launch_bounds__(256) conv_rotary_append_rows_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, uint32_t ld,
                                                                      const __grid_constant__ AttnWindow win, uint32_t heads, uint32_t kv_heads, uint32_t pitch,
                                                                      uint32_t tokens, const int* __restrict__ pos_ptr, float* __restrict__ q_out,
                                                                      float* __restrict__ k_cache, float* __restrict__ v_cache, uint32_t max_positions,
                                                                      int* error_word) {
    pdl_launch_dependents();
    pdl_wait();
    const AttnRotary& ro = win.rotary;
    const int t0 = static_cast<int>(blockIdx.x) * kStrip, n = min(kStrip, static_cast<int>(tokens) - t0), pos = *pos_ptr;
    if (pos < 0 || static_cast<long long>(pos) + tokens > static_cast<long long>(max_positions)) {
        if (threadIdx.x == 0) atomicExch(error_word, kErrBadPosition);
        return;
    }
    const uint32_t lane = threadIdx.x & 31, half = ro.turn.half, items = heads + 2 * kv_heads;
    for (uint32_t item = blockIdx.y * 8 + (threadIdx.x >> 5); item < items; item += gridDim.y * 8) {
        const bool is_q = item < heads, is_k = !is_q && item < heads + kv_heads, is_v = !is_q && !is_k;
        const uint32_t g = is_q ? item : is_k ? item - heads : item - heads - kv_heads, size = is_v ? win.v_dim : win.qk_dim;
        const uint32_t first = is_q ? 0u : is_k ? heads * win.qk_dim : (heads + kv_heads) * win.qk_dim;      // the convolution's channel of the part's first column
        const float* src = (is_q ? q : is_k ? k : v) + g * size;
        const uint32_t c0 = first + g * size, step = (is_q ? heads : kv_heads) * pitch;
        float* dst = is_q ? q_out + (static_cast<size_t>(t0) * heads + g) * pitch : (is_k ? k_cache : v_cache) + (static_cast<size_t>(pos + t0) * kv_heads + g) * pitch;
        float a[kStrip], b[kStrip];
        const uint32_t turned = is_v ? 0u : 2 * half;
        for (uint32_t i = lane; i < turned / 2; i += 32) {
            conv_sum_strip(ro.conv, src + i, ld, t0, n, pos, c0 + i, a);
            conv_sum_strip(ro.conv, src + half + i, ld, t0, n, pos, c0 + half + i, b);
#pragma unroll
            for (int j = 0; j < kStrip; ++j) {
                if (j >= n) break;
                const size_t row = rotation_row(ro.turn, pos + t0 + j) + i;
                const float c = __ldg(ro.turn.cos_t + row), s = __ldg(ro.turn.sin_t + row);
                dst[static_cast<size_t>(j) * step + i] = rotated_low(a[j], b[j], c, s);
                dst[static_cast<size_t>(j) * step + half + i] = rotated_high(a[j], b[j], c, s);
            }
        }
        for (uint32_t i = turned + lane; i < pitch; i += 32) {
#pragma unroll
            for (int j = 0; j < kStrip; ++j) a[j] = 0.0f;
            if (i < size) {
                conv_sum_strip(ro.conv, src + i, ld, t0, n, pos, c0 + i, a);
                if (is_v && (ro.v_first || ro.v_keep)) {
#pragma unroll
                    for (int j = 0; j < kStrip; ++j) {
                        if (j >= n) break;
                        const size_t at = static_cast<size_t>(t0 + j) * kv_heads * size + g * size + i;
                        if (ro.v_first) a[j] = mixed_value(a[j], __ldcg(ro.v_first + at), ro.share);
                        if (ro.v_keep) ro.v_keep[at] = a[j];
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < kStrip; ++j)
                if (j < n) dst[static_cast<size_t>(j) * step + i] = a[j];
        }
    }
}

}  // namespace zk
