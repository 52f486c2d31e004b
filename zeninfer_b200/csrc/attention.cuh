// Grouped-query attention over an fp32 KV cache: one new token (attention_decode_kernel) and a block of new tokens
// (attention_prefill_kernel), each over all earlier positions or a sliding window, optionally with the window's kept first
// tokens and a per-head distance bias.
#pragma once
#include <cooperative_groups.h>

#include <cstdint>

#include "token_mixing.cuh"
#include "zk_ptx.cuh"

namespace zk {

// What forms q, k and v where they are convolved and rotated: channels q | k | v in the convolution's numbering, the rotation of
// q and k, and values mixed with those of an earlier layer: v <- (1 - share) v + share v_first.
struct AttnRotary {
    ShortConv conv;
    HalfRotation turn;
    const float* v_first;     // [tokens][kv_heads][v_dim]: the earlier layer's values of the same tokens; null: no mixing
    float* v_keep;            // where this layer's values go for later layers, or null
    float share;
};

// How attention_decode_kernel<kFused = true> finds q and k_new: to be rotated in adjacent pairs by the tables passed beside them, to be
// RMS-normed per head, or to be convolved and rotated by halves.
enum AttnInput : int { kAttnAdjacentPairs = 0, kAttnNormed = 1, kAttnConvRotary = 2 };

// What a windowed attention with a distance bias adds to the plain one.  Query position i sees key position j <= i when
// i - j < window or j < keep_first; the score is (q . k) * scale - slope_h * (i - j), slope_h = 2^(-8 (h + 1) / heads).
struct AttnWindow {
    uint32_t keep_first;      // kept tokens at the start of the sequence (0: none)
    uint32_t biased;          // 1: the distance bias is taken off the scores
    // kAttnNormed and kAttnConvRotary: q, k and v arrive as raw projections and are finished here, value heads may be narrower
    // than the cache's head pitch, and the output is scaled by a gate.
    const float* q_weight;    // kAttnNormed: [qk_dim]
    const float* k_weight;    // kAttnNormed: [qk_dim]
    const float* gate;        // [heads], or [heads][v_dim] with gate_values: the output is multiplied by its sigmoid; null: no gate
    float eps;
    uint32_t qk_dim, v_dim;   // real sizes of a query/key and a value head; the cache's pitch D covers both, zero-padded
    uint32_t gate_values;
    AttnRotary rotary;        // kAttnConvRotary
};

__device__ __forceinline__ float attn_slope(uint32_t h, uint32_t heads) {
    return static_cast<float>(exp2(-8.0 * static_cast<double>(h + 1) / static_cast<double>(heads)));
}
__device__ __forceinline__ float mixed_value(float v, float first, float share) { return fmaf(share, first, (1.0f - share) * v); }

// Grouped-query attention for one new token.  A cluster of kAttnSplit CTAs serves one query head: CTA `rank` takes
// positions first + rank, first + rank + kAttnSplit, ...; inside a CTA a warp takes a position at a time, four dimensions
// per lane, kAttnUnroll positions in flight.  At a few hundred positions the kernel is bound by memory latency, not
// bandwidth, so it is built to pay as few dependent round trips as possible: the key AND value rows of a warp's
// positions are requested together, and every warp keeps a running maximum m, denominator l and output accumulator
// (the streaming form of the softmax: when a new maximum arrives, l and the accumulator are rescaled by
// exp(m_old - m_new)), so nothing waits for a block-wide maximum between the keys and the values.  Eight warps x four
// positions x eight CTAs cover 256 positions per round (kWide: head dimensions above 128, eight floats per lane).
// Resources are part of the design: the kernel runs between two projection launches that overlap with it, so a CTA
// stays at 256 threads and at most 85 registers.  Measured inside a Llama-3-8B layer at position 575: 8.5 us with four
// positions per warp and 85 registers; 11.2 us with eight positions and 128 registers although that version is the
// faster one when timed alone (6.8 against 8.6 us); 512 threads ran the clusters in two waves (19 us); builds that
// spill to reach 48 or 64 registers lose more than they gain.  The warps' (m, l, accumulator) are merged in shared memory,
// rank 0 merges the CTAs' shares through distributed shared memory:
// out = sum_r w_r out_r / sum_r w_r l_r with w_r = exp(m_r - max m), which is exp(score - max) / denominator applied
// to v, the reference's formula (src/adapters/dense_transformer_runtime.cpp:4284-4337); denominators are kept in double as there.
// D must be a multiple of 4 and at most 256.
constexpr int kAttnThreads = 256;
constexpr int kAttnSplit = 8;
constexpr int kAttnMaxD = 256;

struct AttnShare {          // one CTA's contribution, read by rank 0 of the cluster
    float out[kAttnMaxD];
    float max_score;
    double sum;
};

// One rotation of an adjacent pair, with every product and the sum rounded on its own as in the reference's scalar
// loop (a fused multiply-add here would make a cached key differ in the last bit from the one used in its own step).
__device__ __forceinline__ void rope_pair(float& a, float& b, float c, float s) {
    const float ra = __fsub_rn(__fmul_rn(a, c), __fmul_rn(b, s)), rb = __fadd_rn(__fmul_rn(a, s), __fmul_rn(b, c));
    a = ra; b = rb;
}
// dimensions base .. base+3 of a head vector: pairs base/2 and base/2 + 1 (adjacent pairing)
__device__ __forceinline__ void rope_quad(float4& v, uint32_t base, uint32_t pairs, const float* __restrict__ c, const float* __restrict__ s) {
    const uint32_t pr = base >> 1;
    if (pr < pairs) rope_pair(v.x, v.y, c[pr], s[pr]);
    if (pr + 1 < pairs) rope_pair(v.z, v.w, c[pr + 1], s[pr + 1]);
}

// kFused: q, k_new, v_new are the raw projections of the token in flight; the kernel applies the adjacent-pair rotary
// embedding (host-built table rows of *pos_ptr) to q and k_new in registers, attends to the cache for earlier
// positions and to k_new / v_new for the current one, and the cluster of each KV group's first query head appends the
// rotated key and the value to the caches.  This is the reference's attention_block contract
// (include/zen/d3d12_backend.h:247).  Other clusters never read the cache at the current position, so the append
// races with nothing.
//
// kInput (with kFused): kAttnNormed norms q and k_new per head with AttnWindow's weights instead of the rotation; kAttnConvRotary
// convolves all three, rotates q and k_new by halves and mixes v_new.  In both the kept first tokens and the distance bias of
// AttnWindow apply; out is [heads][v_dim], gated.  The cache's head pitch is D for keys and values alike, zero beyond qk_dim / v_dim.
template <bool kFused, bool kWide, int kInput = kAttnAdjacentPairs>
__global__ void __cluster_dims__(kAttnSplit, 1, 1) __launch_bounds__(kAttnThreads, kWide ? 2 : 3)
    attention_decode_kernel(const float* __restrict__ q, const float* __restrict__ k_cache_in, const float* __restrict__ v_cache_in,
                            const int* __restrict__ pos_ptr, float* __restrict__ out, uint32_t heads, uint32_t kv_heads, uint32_t D, float scale,
                            uint32_t window, uint32_t max_positions, int* error_word, const float* __restrict__ k_new, const float* __restrict__ v_new,
                            const float* __restrict__ cos_t, const float* __restrict__ sin_t, uint32_t pairs, float* k_cache_out, float* v_cache_out,
                            AttnWindow win) {
    constexpr bool kNormed = kInput == kAttnNormed, kOwn = kInput != kAttnAdjacentPairs;    // kOwn: finishes and appends its own key
    static_assert(kFused || !kOwn, "the token in flight is formed here");
    const float* k_cache = kFused ? k_cache_out : k_cache_in;   // fused: the caches are also written here, so no read-only promise
    const float* v_cache = kFused ? v_cache_out : v_cache_in;
    namespace cg = cooperative_groups;
    constexpr int kWarps = kAttnThreads / 32, kAttnUnroll = 4;
    __shared__ AttnShare share;
    __shared__ __align__(16) float partial[kWarps * kAttnMaxD];   // [warp][dimension]: the warps' accumulators
    __shared__ float warp_max[kWarps];
    __shared__ double warp_sum[kWarps];
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t rank = cluster.block_rank();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t h = blockIdx.y, kh = h / (heads / kv_heads), kw = kv_heads * D;
    const bool lo_on = 4u * lane < D, hi_on = kWide && 128u + 4u * lane < D;   // !kWide: the compiler drops the upper halves
    pdl_launch_dependents();
    pdl_wait();
    // the first round trip: the position, and beside it everything whose address does not depend on it
    const int pos = *pos_ptr;
    const uint32_t d_q = kOwn ? win.qk_dim : D, d_v = kOwn ? win.v_dim : D;
    const float* qh = q + static_cast<size_t>(h) * d_q;
    float4 q0 = make_float4(0.f, 0.f, 0.f, 0.f), q1 = q0;
    // real head sizes need not be a multiple of four floats, nor their start in the projection row aligned
    auto ragged = [](const float* v, uint32_t first, uint32_t n) {
        float4 r;
        r.x = first < n ? __ldcg(v + first) : 0.0f;
        r.y = first + 1 < n ? __ldcg(v + first + 1) : 0.0f;
        r.z = first + 2 < n ? __ldcg(v + first + 2) : 0.0f;
        r.w = first + 3 < n ? __ldcg(v + first + 3) : 0.0f;
        return r;
    };
    float gate_value = 1.0f;
    if (kOwn && win.gate) {
        if (!win.gate_values) gate_value = logistic(__ldcg(win.gate + h));
        else if (threadIdx.x < d_v) gate_value = logistic(__ldcg(win.gate + static_cast<size_t>(h) * d_v + threadIdx.x));
    }
    if (kNormed) {
        q0 = ragged(qh, 4 * lane, d_q);
        if (kWide) q1 = ragged(qh, 128 + 4 * lane, d_q);
    }
    if (!kOwn && lo_on) q0 = __ldcg(reinterpret_cast<const float4*>(qh + 4 * lane));      // q, k_new, v_new: written by the launch before this one
    if (!kOwn && hi_on) q1 = __ldcg(reinterpret_cast<const float4*>(qh + 128 + 4 * lane));
    const float* knew = kFused ? k_new + static_cast<size_t>(kh) * d_q : nullptr;
    const float* vnew = kFused ? v_new + static_cast<size_t>(kh) * d_v : nullptr;
    float4 kn0 = make_float4(0.f, 0.f, 0.f, 0.f), kn1 = kn0, vn0 = kn0, vn1 = kn0;   // the token in flight, every warp's copy
    if (kNormed) {
        kn0 = ragged(knew, 4 * lane, d_q);
        vn0 = ragged(vnew, 4 * lane, d_v);
        if (kWide) { kn1 = ragged(knew, 128 + 4 * lane, d_q); vn1 = ragged(vnew, 128 + 4 * lane, d_v); }
        // every warp holds the whole head: its sum of squares is one warp reduction
        auto normed = [&](float4& lo, float4& hi, const float* weight) {
            float ss = lo.x * lo.x + lo.y * lo.y + lo.z * lo.z + lo.w * lo.w + hi.x * hi.x + hi.y * hi.y + hi.z * hi.z + hi.w * hi.w;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float inv = 1.0f / sqrtf(ss / static_cast<float>(d_q) + win.eps);
            const float4 wl = ragged(weight, 4 * lane, d_q);
            lo = make_float4(lo.x * inv * wl.x, lo.y * inv * wl.y, lo.z * inv * wl.z, lo.w * inv * wl.w);
            if (kWide) {
                const float4 wh = ragged(weight, 128 + 4 * lane, d_q);
                hi = make_float4(hi.x * inv * wh.x, hi.y * inv * wh.y, hi.z * inv * wh.z, hi.w * inv * wh.w);
            }
        };
        normed(q0, q1, win.q_weight);
        normed(kn0, kn1, win.k_weight);
    }
    if (kFused && !kOwn) {
        if (lo_on) { kn0 = __ldcg(reinterpret_cast<const float4*>(knew + 4 * lane)); vn0 = __ldcg(reinterpret_cast<const float4*>(vnew + 4 * lane)); }
        if (hi_on) { kn1 = __ldcg(reinterpret_cast<const float4*>(knew + 128 + 4 * lane)); vn1 = __ldcg(reinterpret_cast<const float4*>(vnew + 128 + 4 * lane)); }
    }
    const bool bad = pos < 0 || static_cast<uint32_t>(pos) >= max_positions;
    if constexpr (kInput == kAttnConvRotary) {
        __shared__ __align__(16) float raw[2][kAttnMaxD], head[3][kAttnMaxD];        // q and k convolved; q, k, v of this head finished; zero beyond their sizes
        const AttnRotary& ro = win.rotary;
        const uint32_t i = threadIdx.x, cq = h * d_q + i, ck = (heads + kh) * d_q + i, cv = (heads + kv_heads) * d_q + kh * d_v + i, half = ro.turn.half;
        const bool owner = rank == 0 && h % (heads / kv_heads) == 0, turns = i < 2 * half, is_low = i < half;
        const int at = bad ? 0 : pos;
        float* slot = ro.conv.taps ? ro.conv.ring + static_cast<size_t>(static_cast<uint32_t>(at) % ro.conv.taps) * ro.conv.channels : nullptr;
        float c = 1.0f, s = 0.0f, yq = 0.0f, yk = 0.0f, yv = 0.0f;
        if (turns) {
            const size_t row = rotation_row(ro.turn, at) + (is_low ? i : i - half);
            c = __ldg(ro.turn.cos_t + row);
            s = __ldg(ro.turn.sin_t + row);
        }
        if (!bad && i < d_q) {
            yq = conv_sum(ro.conv, qh + i, 0, 0, at, cq);
            yk = conv_sum(ro.conv, knew + i, 0, 0, at, ck);
            if (slot && rank == 0) slot[cq] = __ldcg(qh + i);
            if (slot && owner) slot[ck] = __ldcg(knew + i);
        }
        if (!bad && i < d_v) {
            yv = conv_sum(ro.conv, vnew + i, 0, 0, at, cv);
            if (ro.v_first) yv = mixed_value(yv, __ldcg(ro.v_first + kh * d_v + i), ro.share);
            if (ro.v_keep && owner) ro.v_keep[kh * d_v + i] = yv;
            if (slot && owner) slot[cv] = __ldcg(vnew + i);
        }
        raw[0][i] = yq;
        raw[1][i] = yk;
        head[2][i] = yv;
        __syncthreads();
        if (turns) {
            const uint32_t other = is_low ? i + half : i - half;
            yq = is_low ? rotated_low(yq, raw[0][other], c, s) : rotated_high(raw[0][other], yq, c, s);
            yk = is_low ? rotated_low(yk, raw[1][other], c, s) : rotated_high(raw[1][other], yk, c, s);
        }
        head[0][i] = yq;
        head[1][i] = yk;
        __syncthreads();
        q0 = *reinterpret_cast<const float4*>(&head[0][4 * lane]);
        kn0 = *reinterpret_cast<const float4*>(&head[1][4 * lane]);
        vn0 = *reinterpret_cast<const float4*>(&head[2][4 * lane]);
        if (kWide) {
            q1 = *reinterpret_cast<const float4*>(&head[0][128 + 4 * lane]);
            kn1 = *reinterpret_cast<const float4*>(&head[1][128 + 4 * lane]);
            vn1 = *reinterpret_cast<const float4*>(&head[2][128 + 4 * lane]);
        }
    }
    if (bad && threadIdx.x == 0 && blockIdx.x == 0 && blockIdx.y == 0) atomicExch(error_word, kErrBadPosition);
    const uint32_t first = (window && static_cast<uint32_t>(pos) + 1 > window) ? static_cast<uint32_t>(pos) + 1 - window : 0u;
    uint32_t kept = 0;                                                                        // kept tokens the window has left behind
    if (kOwn) kept = min(win.keep_first, first);
    const uint32_t count = bad ? 0u : static_cast<uint32_t>(pos) + 1 - first + kept;          // positions attended by the head
    const uint32_t mine = count > rank ? (count - rank + kAttnSplit - 1) / kAttnSplit : 0u;   // ... by this CTA
    const float* kbase = k_cache + static_cast<size_t>(first + rank) * kw + static_cast<size_t>(kh) * D;
    const float* vbase = v_cache + static_cast<size_t>(first + rank) * kw + static_cast<size_t>(kh) * D;
    const size_t step = static_cast<size_t>(kAttnSplit) * kw;     // floats between this CTA's consecutive positions
    const uint32_t last = count ? count - 1 : 0;                  // index of the current position among the attended ones
    const uint32_t skipped = first - kept;                        // positions between the kept tokens and the window
    auto position_of = [&](uint32_t index) { return index < kept ? index : index + skipped; };
    const float slope = kOwn && win.biased ? attn_slope(h, heads) : 0.0f;

    float run_max = -INFINITY;
    double run_sum = 0.0;
    float4 a0 = make_float4(0.f, 0.f, 0.f, 0.f), a1 = a0;
    bool turned = false;
    for (uint32_t i0 = warp; i0 < mine; i0 += kWarps * kAttnUnroll) {
        // the second round trip: keys and values of this round's positions together (and, the first time, the cos/sin row)
        float4 ka[kAttnUnroll], kb[kAttnUnroll], va[kAttnUnroll], vb[kAttnUnroll];
        bool fresh[kAttnUnroll];
#pragma unroll
        for (int u = 0; u < kAttnUnroll; ++u) {
            const uint32_t i = i0 + u * kWarps;
            ka[u] = kb[u] = va[u] = vb[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            fresh[u] = kFused && i < mine && rank + i * kAttnSplit == last;     // the token in flight: not in the cache yet
            if (i < mine && !fresh[u]) {
                const float* kt = kbase + static_cast<size_t>(i) * step;
                const float* vt = vbase + static_cast<size_t>(i) * step;
                if (kOwn) {
                    const size_t row = static_cast<size_t>(position_of(rank + i * kAttnSplit)) * kw + static_cast<size_t>(kh) * D;
                    kt = k_cache + row;
                    vt = v_cache + row;
                }
                if (lo_on) { ka[u] = __ldcg(reinterpret_cast<const float4*>(kt + 4 * lane)); va[u] = __ldcg(reinterpret_cast<const float4*>(vt + 4 * lane)); }
                if (hi_on) { kb[u] = __ldcg(reinterpret_cast<const float4*>(kt + 128 + 4 * lane)); vb[u] = __ldcg(reinterpret_cast<const float4*>(vt + 128 + 4 * lane)); }
            }
        }
        if (kFused && !kOwn && !turned && !bad) {   // rotate q and the new key once (table rows of the current position)
            const float* cs = cos_t + static_cast<size_t>(pos) * pairs;
            const float* sn = sin_t + static_cast<size_t>(pos) * pairs;
            if (lo_on) { rope_quad(q0, 4u * lane, pairs, cs, sn); rope_quad(kn0, 4u * lane, pairs, cs, sn); }
            if (hi_on) { rope_quad(q1, 128u + 4u * lane, pairs, cs, sn); rope_quad(kn1, 128u + 4u * lane, pairs, cs, sn); }
            turned = true;
        }
        float sc[kAttnUnroll];
#pragma unroll
        for (int u = 0; u < kAttnUnroll; ++u) {
            if (fresh[u]) { ka[u] = kn0; kb[u] = kn1; va[u] = vn0; vb[u] = vn1; }
            float acc = q0.x * ka[u].x + q0.y * ka[u].y + q0.z * ka[u].z + q0.w * ka[u].w + q1.x * kb[u].x + q1.y * kb[u].y + q1.z * kb[u].z + q1.w * kb[u].w;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            sc[u] = i0 + u * kWarps < mine ? acc * scale : -INFINITY;
            if (kOwn && i0 + u * kWarps < mine) sc[u] -= slope * static_cast<float>(static_cast<uint32_t>(pos) - position_of(rank + (i0 + u * kWarps) * kAttnSplit));
        }
        float new_max = run_max;
#pragma unroll
        for (int u = 0; u < kAttnUnroll; ++u) new_max = fmaxf(new_max, sc[u]);
        // i0 < mine, so at least sc[0] is a real score; a non-finite maximum (NaN or +inf scores) is caught by the final check
        const float corr = run_max == -INFINITY ? 0.0f : expf(run_max - new_max);
        a0.x *= corr; a0.y *= corr; a0.z *= corr; a0.w *= corr;
        a1.x *= corr; a1.y *= corr; a1.z *= corr; a1.w *= corr;
        double add = 0.0;
#pragma unroll
        for (int u = 0; u < kAttnUnroll; ++u) {
            const float e = sc[u] == -INFINITY ? 0.0f : expf(sc[u] - new_max);
            add += e;
            a0.x += e * va[u].x; a0.y += e * va[u].y; a0.z += e * va[u].z; a0.w += e * va[u].w;
            a1.x += e * vb[u].x; a1.y += e * vb[u].y; a1.z += e * vb[u].z; a1.w += e * vb[u].w;
        }
        run_sum = run_sum * static_cast<double>(corr) + add;
        run_max = new_max;
    }
    // append: the cluster of the KV group's first query head, the CTA that owns the current position
    if (kOwn && !bad && h % (heads / kv_heads) == 0 && rank == last % kAttnSplit && warp == 0) {
        float* kr = k_cache_out + static_cast<size_t>(pos) * kw + static_cast<size_t>(kh) * D;
        float* vr = v_cache_out + static_cast<size_t>(pos) * kw + static_cast<size_t>(kh) * D;
        if (lo_on) { *reinterpret_cast<float4*>(kr + 4 * lane) = kn0; *reinterpret_cast<float4*>(vr + 4 * lane) = vn0; }
        if (hi_on) { *reinterpret_cast<float4*>(kr + 128 + 4 * lane) = kn1; *reinterpret_cast<float4*>(vr + 128 + 4 * lane) = vn1; }
    }
    if (kFused && !kOwn && !bad && h % (heads / kv_heads) == 0 && rank == last % kAttnSplit && threadIdx.x < D) {
        const float* cs = cos_t + static_cast<size_t>(pos) * pairs;
        const float* sn = sin_t + static_cast<size_t>(pos) * pairs;
        const uint32_t dd = threadIdx.x, pr = dd >> 1;
        float a = __ldcg(knew + (dd & ~1u)), b = __ldcg(knew + (dd | 1u));
        if (pr < pairs) rope_pair(a, b, cs[pr], sn[pr]);
        k_cache_out[static_cast<size_t>(pos) * kw + static_cast<size_t>(kh) * D + dd] = (dd & 1u) ? b : a;
        v_cache_out[static_cast<size_t>(pos) * kw + static_cast<size_t>(kh) * D + dd] = __ldcg(vnew + dd);
    }
    // merge the warps: this CTA's (maximum, denominator, output share)
    if (lo_on) *reinterpret_cast<float4*>(&partial[warp * kAttnMaxD + 4 * lane]) = a0;
    if (hi_on) *reinterpret_cast<float4*>(&partial[warp * kAttnMaxD + 128 + 4 * lane]) = a1;
    if (lane == 0) { warp_max[warp] = run_max; warp_sum[warp] = run_sum; }
    __syncthreads();
    float cta_max = warp_max[0];
#pragma unroll
    for (int w = 1; w < kWarps; ++w) cta_max = fmaxf(cta_max, warp_max[w]);
    if (threadIdx.x < D) {
        float total = 0.0f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
            const float wm = warp_max[w];
            if (wm != -INFINITY) total += expf(wm - cta_max) * partial[w * kAttnMaxD + threadIdx.x];
        }
        share.out[threadIdx.x] = total;
    }
    if (threadIdx.x == 0) {
        double sum = 0.0;
        for (int w = 0; w < kWarps; ++w)
            if (warp_max[w] != -INFINITY) sum += static_cast<double>(expf(warp_max[w] - cta_max)) * warp_sum[w];
        share.max_score = cta_max;
        share.sum = sum;
    }
    cluster.sync();                                   // every CTA's share is complete and visible
    if (rank == 0 && !bad) {
        float m = -INFINITY;
        for (uint32_t r = 0; r < kAttnSplit; ++r) m = fmaxf(m, cluster.map_shared_rank(&share, r)->max_score);
        double denom = 0.0;
        float w[kAttnSplit];
        for (uint32_t r = 0; r < kAttnSplit; ++r) {
            const AttnShare* sh = cluster.map_shared_rank(&share, r);
            w[r] = sh->max_score == -INFINITY ? 0.0f : expf(sh->max_score - m);   // a CTA without positions contributes nothing
            denom += static_cast<double>(w[r]) * sh->sum;
        }
        if (!(denom > 0.0) || !isfinite(denom)) {
            if (threadIdx.x == 0) atomicExch(error_word, kErrNonFinite);
        } else if (threadIdx.x < d_v) {
            const float inv = 1.0f / static_cast<float>(denom);
            float total = 0.0f;
            for (uint32_t r = 0; r < kAttnSplit; ++r) total += w[r] * cluster.map_shared_rank(&share, r)->out[threadIdx.x];
            out[static_cast<size_t>(h) * d_v + threadIdx.x] = kOwn ? total * inv * gate_value : total * inv;
        }
    }
    cluster.sync();                                   // nobody leaves while rank 0 still reads its shared memory
}

// Causal grouped-query attention for a block of T new tokens whose keys and values are already in the caches.
// A CTA takes kPfTokens consecutive tokens, one KV head and R query heads of that KV head's group (R = 4, 2 or 1, the
// largest that divides the group and keeps the rows in registers).  A token is held by kPfLanes threads; thread `part`
// owns the float4 columns part, part + kPfLanes, ... of the head and keeps them for all R heads, so a key or value word
// read from shared memory feeds R multiply-adds (shared-memory bandwidth, 128 bytes per clock per SM, bounds this
// kernel otherwise) and the token's threads read consecutive 16-byte words (no bank conflict).  Products and
// accumulations are packed fp32 pairs (fma.rn.f32x2: each half is an IEEE fused multiply-add).  Keys and values come
// through shared memory in blocks of kPfBlock positions; the softmax is the running-maximum form (out and denominator
// rescaled when the maximum moves), which equals the reference's two-pass form up to rounding (attention rows of
// forward_batch, :3041-3570).  Token t attends positions [first, pos0 + t], first = the sliding-window start or 0.
// The grid is one-dimensional and ordered by work: the tiles of the last tokens (the longest key ranges) take the low
// block indices and start first.
#ifndef ZK_PF_STEP
#define ZK_PF_STEP 4
#endif
constexpr int kPfTokens = 16, kPfLanes = 8, kPfBlock = 32, kPfThreads = kPfTokens * kPfLanes, kPfStep = ZK_PF_STEP;
static_assert(kPfBlock % kPfStep == 0, "a round of positions must not straddle two staged blocks");
// 16-byte asynchronous copy global -> shared (bypassing L1); `bytes` = 16, or 0 for a zero fill.
__device__ __forceinline__ void cp_async_16(float* smem_dst, const float* gmem_src, uint32_t bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(gmem_src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int kPending>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(kPending) : "memory"); }
__device__ __forceinline__ uint64_t pf_pack(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void pf_unpack(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t pf_fma(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t pf_mul(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
// The lane (within a token's kPfLanes) that ends the score reduction with head r's sum and keeps that row's softmax state.
template <int R>
__device__ __forceinline__ constexpr int pf_owner(int r) { return R == 4 ? ((r >> 1) * 4 + (r & 1) * 2) : R == 2 ? r * 4 : 0; }
//
// kWindowed: AttnWindow's kept first tokens and distance bias.  The key blocks then run over the kept tokens the window of the
// tile's first token has left behind, and after them over the window as before.
template <int D, int R, bool kWindowed = false>   // head dimension (a multiple of 32 up to 256) and query heads per thread: compile-time, so the rows stay in registers
__global__ void __launch_bounds__(kPfThreads) attention_prefill_kernel(const float* __restrict__ q, const float* __restrict__ k_cache,
                                                                        const float* __restrict__ v_cache, const int* __restrict__ pos_ptr,
                                                                        float* __restrict__ out, uint32_t tokens, uint32_t heads, uint32_t kv_heads,
                                                                        float scale, uint32_t window, uint32_t max_positions, int* error_word, AttnWindow win) {
    extern __shared__ __align__(16) float kv_smem[];      // two buffers of [2][kPfBlock][D]: keys, then values
    pdl_launch_dependents();
    pdl_wait();
    const int pos0 = *pos_ptr;
    if (pos0 < 0 || static_cast<uint32_t>(pos0) + tokens > max_positions) {
        if (threadIdx.x == 0 && blockIdx.x == 0) atomicExch(error_word, kErrBadPosition);
        return;
    }
    const uint32_t group = heads / kv_heads, passes = group / R, kw = kv_heads * D, qw = heads * D;
    const uint32_t per_tile = kv_heads * passes, n_tiles = gridDim.x / per_tile;
    const uint32_t tile = n_tiles - 1 - blockIdx.x / per_tile, rem = blockIdx.x % per_tile;
    const uint32_t kh = rem / passes, h0 = kh * group + (rem % passes) * R;      // this CTA's heads: h0 .. h0 + R - 1
    constexpr int per4 = D / (4 * kPfLanes);                          // float4 columns per thread and head
    const uint32_t t0 = tile * kPfTokens;
    const uint32_t t_end = min(tokens, t0 + kPfTokens);
    // the span of positions any token of this CTA attends
    const uint32_t last_pos = static_cast<uint32_t>(pos0) + t_end - 1;
    const uint32_t first_any = (window && static_cast<uint32_t>(pos0) + t0 + 1 > window) ? static_cast<uint32_t>(pos0) + t0 + 1 - window : 0u;
    const uint32_t t = t0 + threadIdx.x / kPfLanes, part = threadIdx.x % kPfLanes;
    const bool live = t < t_end;
    const uint32_t my_last = static_cast<uint32_t>(pos0) + t;
    const uint32_t my_first = (window && my_last + 1 > window) ? my_last + 1 - window : 0u;
    uint64_t q01[R][per4], q23[R][per4], a01[R][per4], a23[R][per4];
    // The softmax state of a row lives in one lane: the score reduction below leaves the token's lane `part` with the
    // full sum of one head (head ((part >> 2) << 1 | ((part >> 1) & 1)) for R == 4, part >> 2 for R == 2), and that lane
    // keeps the row's running maximum and denominator.
    float m = -INFINITY;
    double l = 0.0;
#pragma unroll
    for (int r = 0; r < R; ++r) {
#pragma unroll
        for (int i = 0; i < per4; ++i) { q01[r][i] = q23[r][i] = a01[r][i] = a23[r][i] = pf_pack(0.0f, 0.0f); }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float4* qrow = reinterpret_cast<const float4*>(q + static_cast<size_t>(t) * qw + static_cast<size_t>(h0 + r) * D) + part;
#pragma unroll
            for (int i = 0; i < per4; ++i) {
                const float4 v = qrow[i * kPfLanes];
                q01[r][i] = pf_pack(v.x, v.y);
                q23[r][i] = pf_pack(v.z, v.w);
            }
        }
    }
    // Blocks of kPfBlock positions go through two shared-memory buffers: the asynchronous copies of block b + 1 are in
    // flight while block b is consumed.  Rows past last_pos are filled with zeros (a copy of source size 0).
    const uint32_t kept_end = kWindowed ? min(win.keep_first, first_any) : 0u;
    float slope = 0.0f;
    if (kWindowed && win.biased) slope = attn_slope(h0 + (R == 4 ? ((part >> 2) << 1 | ((part >> 1) & 1)) : R == 2 ? part >> 2 : 0u), heads);
    auto stage = [&](uint32_t p0, uint32_t buf) {
        const uint32_t part_last = kWindowed && p0 < kept_end ? kept_end - 1 : last_pos;   // last row of the part the block lies in
        float* kd = kv_smem + buf * (2 * kPfBlock * D);
        float* vd = kd + kPfBlock * D;
#pragma unroll 4
        for (uint32_t i = threadIdx.x; i < kPfBlock * D / 4; i += kPfThreads) {
            const uint32_t row = i / (D / 4), col = i % (D / 4), pos = min(p0 + row, part_last);
            const uint32_t bytes = p0 + row <= part_last ? 16u : 0u;
            const size_t off = static_cast<size_t>(pos) * kw + static_cast<size_t>(kh) * D + col * 4;
            cp_async_16(kd + i * 4, k_cache + off, bytes);
            cp_async_16(vd + i * 4, v_cache + off, bytes);
        }
        cp_async_commit();
    };
    auto next_block = [&](uint32_t p0) { return kWindowed && p0 < kept_end && p0 + kPfBlock >= kept_end ? first_any : p0 + kPfBlock; };
    const uint32_t start = kWindowed && kept_end ? 0u : first_any;
    stage(start, 0);
    uint32_t buf = 0;
    for (uint32_t p0 = start, p_next; p0 <= last_pos; p0 = p_next, buf ^= 1u) {
        p_next = next_block(p0);
        const bool more = p_next <= last_pos;
        if (more) stage(p_next, buf ^ 1u);       // its buffer was read during the previous block, which ended with a barrier
        if (more) cp_async_wait<1>(); else cp_async_wait<0>();
        __syncthreads();
        const float* ks = kv_smem + buf * (2 * kPfBlock * D);
        const float* vs = ks + kPfBlock * D;
        const uint32_t part_last = kWindowed && p0 < kept_end ? kept_end - 1 : last_pos;
        const uint32_t j_end = min(static_cast<uint32_t>(kPfBlock), part_last - p0 + 1);
        // kPfStep positions per round: their score chains, reductions and exponentials are independent of one another, which
        // is what hides the arithmetic and shuffle latencies at the two or three warps per scheduler the row registers allow.
        // Rows of the staged block past last_pos are zeros and fall outside every token's range.
        for (uint32_t j = 0; j < j_end; j += kPfStep) {
            bool in_range[kPfStep];
            bool any = false;
#pragma unroll
            for (int u = 0; u < kPfStep; ++u) {
                const uint32_t pos = p0 + j + u;
                in_range[u] = live && pos >= my_first && pos <= my_last;      // uniform over the token's kPfLanes threads
                if (kWindowed) in_range[u] = live && (pos >= my_first || pos < win.keep_first) && pos <= min(my_last, part_last);
                any |= in_range[u];
            }
            if (!__any_sync(0xffffffffu, any)) continue;                          // none of this warp's tokens attends these positions
            const float4* krow = reinterpret_cast<const float4*>(ks + j * D) + part;
            uint64_t d[kPfStep][R];
#pragma unroll
            for (int u = 0; u < kPfStep; ++u) {
#pragma unroll
                for (int r = 0; r < R; ++r) d[u][r] = pf_pack(0.0f, 0.0f);
            }
#pragma unroll
            for (int i = 0; i < per4; ++i) {
#pragma unroll
                for (int u = 0; u < kPfStep; ++u) {
                    const float4 kk = krow[u * (D / 4) + i * kPfLanes];
                    const uint64_t k01 = pf_pack(kk.x, kk.y), k23 = pf_pack(kk.z, kk.w);
#pragma unroll
                    for (int r = 0; r < R; ++r) d[u][r] = pf_fma(q23[r][i], k23, pf_fma(q01[r][i], k01, d[u][r]));
                }
            }
            // Sum over the token's eight lanes, halving the rows a lane carries at each exchange: lane `part` ends with
            // the full score of its head (R + 1 or 3 shuffles, where one reduction per row would take 3 R).
            float sc[kPfStep];
#pragma unroll
            for (int u = 0; u < kPfStep; ++u) {
                float dot[R];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float d0, d1;
                    pf_unpack(d[u][r], d0, d1);
                    dot[r] = d0 + d1;
                }
                float red;
                if constexpr (R == 4) {
                    const bool hi = part & 4, hi2 = part & 2;
                    float k0 = hi ? dot[2] : dot[0], k1 = hi ? dot[3] : dot[1];
                    k0 += __shfl_xor_sync(0xffffffffu, hi ? dot[0] : dot[2], 4);
                    k1 += __shfl_xor_sync(0xffffffffu, hi ? dot[1] : dot[3], 4);
                    red = (hi2 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, hi2 ? k0 : k1, 2);
                } else if constexpr (R == 2) {
                    const bool hi = part & 4;
                    red = (hi ? dot[1] : dot[0]) + __shfl_xor_sync(0xffffffffu, hi ? dot[0] : dot[1], 4);
                    red += __shfl_xor_sync(0xffffffffu, red, 2);
                } else {
                    red = dot[0] + __shfl_xor_sync(0xffffffffu, dot[0], 4);
                    red += __shfl_xor_sync(0xffffffffu, red, 2);
                }
                red += __shfl_xor_sync(0xffffffffu, red, 1);
                sc[u] = red * scale;
                if (kWindowed) sc[u] -= slope * static_cast<float>(static_cast<int>(my_last) - static_cast<int>(p0 + j + u));
            }
            float m_new = m;
#pragma unroll
            for (int u = 0; u < kPfStep; ++u) m_new = in_range[u] ? fmaxf(m_new, sc[u]) : m_new;
            const bool moved = m_new > m;
            if (__any_sync(0xffffffffu, moved)) {                   // a maximum moves: rescale what has been summed (rare after the first positions)
                const float f = moved ? expf(m - m_new) : 1.0f;     // exp(-inf) = 0 on the first position
                l *= f;
                m = m_new;
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float fr = __shfl_sync(0xffffffffu, f, pf_owner<R>(r), kPfLanes);
                    const uint64_t f2 = pf_pack(fr, fr);
#pragma unroll
                    for (int i = 0; i < per4; ++i) { a01[r][i] = pf_mul(a01[r][i], f2); a23[r][i] = pf_mul(a23[r][i], f2); }
                }
            }
            uint64_t e2[kPfStep][R];
            float e_sum = 0.0f;                                         // the round's terms in fp32, one double addition per round
#pragma unroll
            for (int u = 0; u < kPfStep; ++u) {
                const float e = in_range[u] ? expf(sc[u] - m) : 0.0f;   // a token that does not attend the position adds 0 x value
                e_sum += e;
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float er = __shfl_sync(0xffffffffu, e, pf_owner<R>(r), kPfLanes);
                    e2[u][r] = pf_pack(er, er);
                }
            }
            l += e_sum;
            const float4* vrow = reinterpret_cast<const float4*>(vs + j * D) + part;
#pragma unroll
            for (int i = 0; i < per4; ++i) {
#pragma unroll
                for (int u = 0; u < kPfStep; ++u) {
                    const float4 vv = vrow[u * (D / 4) + i * kPfLanes];
                    const uint64_t v01 = pf_pack(vv.x, vv.y), v23 = pf_pack(vv.z, vv.w);
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        a01[r][i] = pf_fma(e2[u][r], v01, a01[r][i]);
                        a23[r][i] = pf_fma(e2[u][r], v23, a23[r][i]);
                    }
                }
            }
        }
        __syncthreads();                                    // the block's rows are no longer read: the next copies may land in this buffer
    }
    // every lane of the warp takes part in the exchanges below; only live tokens store
    const bool bad = live && (!(l > 0.0) || !isfinite(l));
    const float inv_mine = (live && !bad) ? 1.0f / static_cast<float>(l) : 0.0f;
    if (bad) atomicExch(error_word, kErrNonFinite);
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const float inv = __shfl_sync(0xffffffffu, inv_mine, pf_owner<R>(r), kPfLanes);
        if (live && inv != 0.0f) {
            float4* orow = reinterpret_cast<float4*>(out + static_cast<size_t>(t) * qw + static_cast<size_t>(h0 + r) * D) + part;
#pragma unroll
            for (int i = 0; i < per4; ++i) {
                float4 o;
                pf_unpack(a01[r][i], o.x, o.y);
                pf_unpack(a23[r][i], o.z, o.w);
                o.x *= inv; o.y *= inv; o.z *= inv; o.w *= inv;
                orow[i * kPfLanes] = o;
            }
        }
    }
}

}  // namespace zk
