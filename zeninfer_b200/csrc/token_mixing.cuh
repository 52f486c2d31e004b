// Per-channel pieces the attention and matrix-state mixers share: gates, the short causal convolution over time with its ring of
// earlier inputs, and the rotation of a head's two halves by the token's position.
#pragma once
#include <cstdint>

#include "zk_ptx.cuh"

namespace zk {

__device__ __forceinline__ float logistic(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z * logistic(z); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z + log1pf(expf(-z)) : log1pf(expf(z)); }

// The inputs of the last `taps` tokens are kept in a ring [taps][channels] whose slot is the position modulo taps: a token reads
// the taps - 1 slots before its own and nobody else writes those, so the ring needs no second buffer.
struct ShortConv {
    const float* w;       // [taps][channels]
    float* ring;          // [taps][channels]
    uint32_t taps;        // 0: no convolution
    uint32_t channels;
};

// y = sum_j w_j u(pos + t - taps + 1 + j) of channel c.  x: the channel's inputs at the block's rows (pitch ld); rows before the
// block come from the ring, tokens before the sequence's start are zeros.
__device__ __forceinline__ float conv_sum(const ShortConv& conv, const float* __restrict__ x, uint32_t ld, int t, int pos, uint32_t c) {
    const int taps = static_cast<int>(conv.taps);
    if (taps == 0) return __ldcg(x + static_cast<size_t>(t) * ld);
    float y = 0.0f;
#pragma unroll 4
    for (int j = 0; j < taps; ++j) {
        const int s = t - (taps - 1 - j), at = pos + s;
        const float* src = s >= 0 ? x + static_cast<size_t>(s) * ld : conv.ring + static_cast<size_t>(static_cast<uint32_t>(max(at, 0)) % conv.taps) * conv.channels + c;
        const float v = at >= 0 ? __ldcg(src) : 0.0f;
        y = fmaf(__ldg(conv.w + static_cast<size_t>(j) * conv.channels + c), v, y);
    }
    return y;
}

constexpr int kStrip = 8;          // tokens a warp takes at a time: a channel's inputs stay in registers while the taps slide over them
constexpr int kMaxSlidingTaps = 4; // more taps than this are read again for every token

// y[i] = conv_sum of channel c at tokens t0 .. t0 + n - 1 (n <= kStrip; the rest is not used).
__device__ __forceinline__ void conv_sum_strip(const ShortConv& conv, const float* __restrict__ x, uint32_t ld, int t0, int n, int pos, uint32_t c, float (&y)[kStrip]) {
    const int taps = static_cast<int>(conv.taps);
    if (taps > kMaxSlidingTaps || taps == 0) {
#pragma unroll
        for (int i = 0; i < kStrip; ++i)
            if (i < n) y[i] = conv_sum(conv, x, ld, t0 + i, pos, c);
        return;
    }
    float w[kMaxSlidingTaps], in[kMaxSlidingTaps - 1 + kStrip];       // w right-aligned: the last is the current token's; in[kMaxSlidingTaps - 1 + i]: token t0 + i
#pragma unroll
    for (int j = 0; j < kMaxSlidingTaps; ++j) {
        const int tap = j - (kMaxSlidingTaps - taps);
        w[j] = tap >= 0 ? __ldg(conv.w + static_cast<size_t>(tap) * conv.channels + c) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < kMaxSlidingTaps - 1 + kStrip; ++i) {
        const int s = t0 + i - (kMaxSlidingTaps - 1), at = pos + s;   // block row, position
        in[i] = 0.0f;
        if (at >= 0 && s >= t0 - (taps - 1) && s < t0 + n)
            in[i] = __ldcg(s >= 0 ? x + static_cast<size_t>(s) * ld : conv.ring + static_cast<size_t>(static_cast<uint32_t>(at) % conv.taps) * conv.channels + c);
    }
#pragma unroll
    for (int i = 0; i < kStrip; ++i) {
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < kMaxSlidingTaps; ++j) sum = fmaf(w[j], in[i + j], sum);
        y[i] = sum;
    }
}

// Rotation by position: dimension i < half and its partner i + half turn by the angle of pair i; dimensions from 2 half on pass.
// The angles' cosines and sines come from host-built tables [positions][half].
struct HalfRotation {
    const float* cos_t;
    const float* sin_t;
    uint32_t half;        // 0: no rotation
    uint32_t positions;   // rows of the tables
};
__device__ __forceinline__ size_t rotation_row(const HalfRotation& r, int pos) {     // a position past the tables reads their last row
    return static_cast<size_t>(min(static_cast<uint32_t>(max(pos, 0)), r.positions - 1)) * r.half;
}
__device__ __forceinline__ float rotated_low(float u, float v, float c, float s) { return u * c - v * s; }
__device__ __forceinline__ float rotated_high(float u, float v, float c, float s) { return v * c + u * s; }
// Dimension d of the rotated head vector whose dimension i is x(i); row = rotation_row of its position.
template <typename X>
__device__ __forceinline__ float rotated(const HalfRotation& r, const X& x, uint32_t d, size_t row) {
    if (d >= 2 * r.half) return x(d);
    const bool low = d < r.half;
    const uint32_t i = low ? d : d - r.half;
    const float u = x(i), v = x(i + r.half), c = __ldg(r.cos_t + row + i), s = __ldg(r.sin_t + row + i);
    return low ? rotated_low(u, v, c, s) : rotated_high(u, v, c, s);
}

}  // namespace zk
