// Mixers with a matrix state per head, S [dim][vdim] in fp32, carried from token to token:
//
//   delta rule    S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (g per key channel)
//   gated write   S <- f * S + (1 - f) v^T;           o = S^T q                       (f per key channel, no key)
//   decayed write S <- g * S + k v^T;                 o = S^T q                       (g per key channel of the token, or one constant
//                                                                                      per head; q and k may be rotated by position)
//
// state_scan_kernel walks a block of tokens, eight at a time, with the state in registers; state_step_kernel takes one token and
// does everything between the layer's input projections and its output projection.  The kernels around the scan form its inputs (short causal
// convolution, unit norms, decays, gates) for all tokens at once.
//
// Device layout of a state: [heads][vdim][pitch], pitch = dim rounded up to 32 and zero beyond dim, so that eight lanes read a
// column's rows as consecutive 16-byte words.
#pragma once
#include "gemv_bf16.cuh"
#include "token_mixing.cuh"

namespace zk {

constexpr float kUnitEps = 1e-6f;
enum StateRule : int { kGatedWrite = 0, kDeltaRule = 1, kDecayedWrite = 2 };

struct LinearLayer {
    uint32_t heads, kv_heads, dim, vdim, pitch;
    uint32_t rank_a, rank_g;       // ranks of the decay's (delta rule, decayed write) and the output gate's (delta rule) projections
    uint32_t a2_ld, g2_ld;
    ShortConv conv;                // delta rule: q, k, v channels
    const float* a_log;            // delta rule: [heads]
    const float* dt_bias;          // [heads][dim], added to the decay's projection
    const __nv_bfloat16* a2;       // [heads dim][a2_ld]
    const __nv_bfloat16* g2;       // [heads vdim][g2_ld]
    const float* decay;            // decayed write: [heads] constants, or null: g = sigmoid(a2 a1 + dt_bias)^inv_tau
    float inv_tau;
    HalfRotation turn;             // decayed write: of q and k
    const float* f_bias;           // gated write: [heads][dim]
    const float* lower;            // gated write: [heads][dim]
    const float* norm;             // [vdim]
    float* state;                  // [heads][vdim][pitch]
    float eps;
};
__host__ __device__ inline uint32_t linear_channels(const LinearLayer& l) { return 2 * l.kv_heads * l.dim + l.heads * l.vdim; }
__device__ __forceinline__ float channel_decay(float z, float inv_tau) { return expf(-softplus_f(-z) * inv_tau); }     // sigmoid(z)^inv_tau

// ---- inputs of the scan for a block of tokens -------------------------------------------------------------------------

// Delta rule.  proj [T][ld]: q | k | v | b columns; decay [T][heads dim] = W_a2 W_a1 h.
//   q, k [T][kv_heads][pitch] unit vectors (q also times dim^-1/2), g [T][heads][pitch], v [T][heads vdim], beta [T][heads].
// A warp takes (strip of tokens, item): a q or k head, 32 value channels, or a head's decays.  Grid: (strips, CTAs that share one).
__global__ void __launch_bounds__(256) delta_inputs_rows_kernel(const __grid_constant__ LinearLayer l, const float* __restrict__ proj, uint32_t ld, uint32_t tokens,
                                                                const float* __restrict__ decay, uint32_t decay_ld, const int* __restrict__ pos_ptr,
                                                                float* __restrict__ q, float* __restrict__ k, float* __restrict__ g, float* __restrict__ v,
                                                                float* __restrict__ beta) {
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = static_cast<int>(blockIdx.x) * kStrip, n = min(kStrip, static_cast<int>(tokens) - t0), pos = *pos_ptr;
    const uint32_t lane = threadIdx.x & 31, channels = linear_channels(l), kd = l.kv_heads * l.dim, nv = l.heads * l.vdim;
    auto silu_strip = [&](uint32_t c, float (&y)[kStrip]) {
        conv_sum_strip(l.conv, proj + c, ld, t0, n, pos, c, y);
#pragma unroll
        for (int i = 0; i < kStrip; ++i) y[i] = silu_f(y[i]);
    };
    const uint32_t qk_items = 2 * l.kv_heads, v_items = (nv + 31) / 32, items = qk_items + v_items + l.heads;
    for (uint32_t item = blockIdx.y * 8 + (threadIdx.x >> 5); item < items; item += gridDim.y * 8) {
        float y[kStrip];
        if (item < qk_items) {
            const bool is_q = item < l.kv_heads;
            const uint32_t head = is_q ? item : item - l.kv_heads, c0 = (is_q ? 0u : kd) + head * l.dim;
            float* dst = (is_q ? q : k) + (static_cast<size_t>(t0) * l.kv_heads + head) * l.pitch;
            const float scale = is_q ? 1.0f / sqrtf(static_cast<float>(l.dim)) : 1.0f;
            float ss[kStrip], last[kStrip];      // last: the head's final 32 channels, which need not go out unscaled
#pragma unroll
            for (int i = 0; i < kStrip; ++i) ss[i] = last[i] = 0.0f;
            for (uint32_t d = lane; d < l.pitch; d += 32) {            // unscaled first: a lane reads back only what it wrote
                const bool more = d + 32 < l.pitch;
#pragma unroll
                for (int i = 0; i < kStrip; ++i) y[i] = 0.0f;
                if (d < l.dim) silu_strip(c0 + d, y);
#pragma unroll
                for (int i = 0; i < kStrip; ++i) {
                    ss[i] += y[i] * y[i];
                    last[i] = y[i];
                    if (more && i < n) dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + d] = y[i];
                }
            }
#pragma unroll
            for (int i = 0; i < kStrip; ++i) ss[i] = scale / sqrtf(warp_sum(ss[i]) + kUnitEps);
            for (uint32_t d = lane; d + 32 < l.pitch; d += 32) {
                float back[kStrip];
#pragma unroll
                for (int i = 0; i < kStrip; ++i) back[i] = i < n ? dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + d] : 0.0f;
#pragma unroll
                for (int i = 0; i < kStrip; ++i)
                    if (i < n) dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + d] = back[i] * ss[i];
            }
#pragma unroll
            for (int i = 0; i < kStrip; ++i)
                if (i < n) dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + l.pitch - 32 + lane] = last[i] * ss[i];
        } else if (item < qk_items + v_items) {
            const uint32_t c = (item - qk_items) * 32 + lane;
            if (c >= nv) continue;
            silu_strip(2 * kd + c, y);
#pragma unroll
            for (int i = 0; i < kStrip; ++i)
                if (i < n) v[static_cast<size_t>(t0 + i) * nv + c] = y[i];
        } else {
            const uint32_t h = item - qk_items - v_items;
            const float rate = -expf(l.a_log[h]);
            for (uint32_t d = lane; d < l.pitch; d += 32) {
                const float bias = d < l.dim ? __ldg(l.dt_bias + h * l.dim + d) : 0.0f;
#pragma unroll
                for (int i = 0; i < kStrip; ++i) y[i] = d < l.dim && i < n ? __ldcg(decay + static_cast<size_t>(t0 + i) * decay_ld + h * l.dim + d) : 0.0f;
#pragma unroll
                for (int i = 0; i < kStrip; ++i)
                    if (i < n) g[(static_cast<size_t>(t0 + i) * l.heads + h) * l.pitch + d] = d < l.dim ? expf(rate * softplus_f(y[i] + bias)) : 0.0f;
            }
            if (static_cast<int>(lane) < n) beta[static_cast<size_t>(t0 + lane) * l.heads + h] = logistic(__ldcg(proj + static_cast<size_t>(t0 + lane) * ld + channels + h));
        }
    }
}

// Gated write.  proj [T][ld]: q | f columns.  q, f [T][heads][pitch]; f = 1 beyond dim (the padding neither decays nor writes).
__global__ void __launch_bounds__(256) gated_write_inputs_rows_kernel(const __grid_constant__ LinearLayer l, const float* __restrict__ proj, uint32_t ld,
                                                                      float* __restrict__ q, float* __restrict__ f) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    for (uint32_t i = threadIdx.x; i < l.heads * l.pitch; i += 256) {
        const uint32_t h = i / l.pitch, d = i % l.pitch, c = h * l.dim + d;
        float qv = 0.0f, fv = 1.0f;
        if (d < l.dim) {
            qv = silu_f(proj[t * ld + c]);
            fv = l.lower[c] + (1.0f - l.lower[c]) * logistic(proj[t * ld + l.heads * l.dim + c] + l.f_bias[c]);
        }
        q[t * l.heads * l.pitch + i] = qv;
        f[t * l.heads * l.pitch + i] = fv;
    }
}

// ---- the scan --------------------------------------------------------------------------------------------------------
//
// Eight tokens at a time.  With S the state before a group and G_t = g_1 ... g_t (channel by channel), unrolling the recurrence gives
//
//   u_t = beta_t (v_t - (k_t G_t) . S - sum_{s<t} A_ts u_s)      A_ts = sum_d k_t k_s g_{s+1} ... g_t
//   o_t = (q_t G_t) . S + sum_{s<=t} B_ts u_s                    B_ts = sum_d q_t k_s g_{s+1} ... g_t
//   S  <- G_8 S + sum_s (k_s g_{s+1} ... g_8) u_s
//
// so that all products with S of a group are independent of one another, and what is sequential is an 8 x 8 triangular system:
// u = T (v - (k G) . S) with T = (1 + diag(beta) A)^-1 diag(beta).  Only products of decays appear, never a quotient, so nothing
// overflows however strong they are.  state_groups_kernel forms, for every group and head at once, the scaled vectors and the
// small matrices T and M (o_t = (q_t G_t) . S + sum_s M_ts w_s with w = v - (k G) . S, M = B T); state_scan_kernel walks the groups.
// The gated write has u = v and k = 1 - f, the decayed write u = v: no T, and M = B.  For the decayed write q and k are columns of the
// projection rows (pitch v_ld, heads of `dim`), and this kernel rotates them and forms the decays.
//
// A group's record, fp32: [k G: 8 x pitch, delta rule only] [q G: 8 x pitch] [k g...: 8 x pitch] [G_8: pitch] [T: 8 x 8, delta only]
// [M: 8 x 8].  Missing tokens at the end of a block have g = 1, k = q = beta = 0 and leave the state as it is.

struct ScanParams {
    const float* q;        // [T][q_heads][pitch]; decayed write: [T][v_ld]
    const float* k;        // [T][q_heads][pitch], delta rule; [T][v_ld], decayed write
    const float* g;        // [T][heads][pitch]; not for the decayed write
    const float* v;        // [T][v_ld], head h's values at column h * vdim
    const float* beta;     // [T][heads]; delta rule only
    const float* low;      // decayed write without constant decays: [T][v_ld], the decay's low-rank inputs
    const int* pos;        // decayed write with a rotation
    float* records;        // [groups][heads][record]
    float* state;          // [heads][vdim][pitch]
    float* out;            // [T][heads][vdim]
    uint32_t tokens, heads, q_heads, vdim, v_ld;
};

constexpr int kGroup = 8;                                                    // tokens per group
constexpr int kScanThreads = 128, kScanColumns = 32, kScanStages = 4;       // columns of S per CTA; groups in flight
__host__ __device__ constexpr uint32_t scan_record_floats(uint32_t pitch, bool delta) { return (delta ? 25 : 17) * pitch + (delta ? 128 : 64); }
template <int kQuads, bool kDelta>
__host__ __device__ constexpr uint32_t scan_smem_bytes() {
    return (kScanStages * (scan_record_floats(kQuads * 32, kDelta) + kGroup * kScanColumns) + (kScanThreads / 32) * kGroup * 8) * 4;
}

// 64 values per lane -> their sums over the warp, two per lane: lane l keeps values 2 l and 2 l + 1.
__device__ __forceinline__ void warp_sum64(float (&v)[64], int lane) {
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
        const bool hi = lane & o;
#pragma unroll
        for (int i = 0; i < 2 * o; ++i) v[i] = (hi ? v[i + 2 * o] : v[i]) + __shfl_xor_sync(0xffffffffu, hi ? v[i] : v[i + 2 * o], o);
    }
}

// One warp per (group, head); a lane takes channels lane, lane + 32, ...  Grid: ceil(groups * heads / 4).
template <int kQuads, int kRule>
__global__ void __launch_bounds__(128) state_groups_kernel(const __grid_constant__ ScanParams p, const __grid_constant__ LinearLayer l) {
    constexpr bool kDelta = kRule == kDeltaRule;
    constexpr uint32_t kPitch = kQuads * 32, kRecord = scan_record_floats(kPitch, kDelta);
    __shared__ float sums[4][64], t_matrix[4][64];
    extern __shared__ __align__(16) float group_low[];          // decayed write: [warp][token][rank rounded up to 8]
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t groups = (p.tokens + kGroup - 1) / kGroup, item = blockIdx.x * 4 + warp;
    if (item >= groups * p.heads) return;                       // whole warps leave; there is no block barrier below
    const uint32_t h = item % p.heads, t0 = item / p.heads * kGroup, qh = h / (p.heads / p.q_heads);
    float* rec = p.records + static_cast<size_t>(item) * kRecord;
    float* const q_out = rec + (kDelta ? 8 * kPitch : 0);
    float* const k_out = q_out + 8 * kPitch;
    float* const g_out = k_out + 8 * kPitch;
    const uint32_t low_ld = (l.rank_a + 7) & ~7u;
    float* const low = group_low + warp * kGroup * low_ld;
    const bool ranked = kRule == kDecayedWrite && !l.decay;
    const float fixed = kRule == kDecayedWrite && l.decay ? __ldg(l.decay + h) : 0.0f, q_scale = 1.0f / sqrtf(static_cast<float>(l.dim));
    const int pos = kRule == kDecayedWrite && l.turn.half ? *p.pos : 0;
    if (ranked) {
        for (uint32_t i = lane; i < kGroup * low_ld; i += 32) {
            const uint32_t t = i / low_ld, c = i % low_ld;
            low[i] = t0 + t < p.tokens && c < l.rank_a ? __ldcg(p.low + static_cast<size_t>(t0 + t) * p.v_ld + c) : 0.0f;
        }
        __syncwarp();
    }
    // entry of (t, s): A's at t (t - 1) / 2 + s for s < t, B's at 28 + t (t + 1) / 2 + s for s <= t
    float acc[64];
#pragma unroll
    for (int i = 0; i < 64; ++i) acc[i] = 0.0f;
#pragma unroll 1
    for (int j = 0; j < kQuads; ++j) {
        const uint32_t d = lane + 32 * j;
        float g[kGroup], k[kGroup], q[kGroup];
        if constexpr (kRule == kDecayedWrite) {
            // every load of a phase is unconditional (tokens past the block read its last one), so that all of them are in flight together
            const bool real = d < l.dim, turns = d < 2 * l.turn.half, is_low = d < l.turn.half;
            auto row_of = [&](int t) { return static_cast<size_t>(min(t0 + t, p.tokens - 1)) * p.v_ld + h * l.dim; };
#pragma unroll
            for (int t = 0; t < kGroup; ++t) {
                q[t] = __ldcg(p.q + row_of(t) + (real ? d : 0u));
                k[t] = __ldcg(p.k + row_of(t) + (real ? d : 0u));
            }
            if (l.turn.half) {
                const uint32_t other = !turns ? 0u : is_low ? d + l.turn.half : d - l.turn.half, pair = !turns ? 0u : is_low ? d : d - l.turn.half;
                float qo[kGroup], ko[kGroup], c[kGroup], s[kGroup];
#pragma unroll
                for (int t = 0; t < kGroup; ++t) {
                    const size_t row = rotation_row(l.turn, pos + static_cast<int>(t0 + t)) + pair;
                    qo[t] = __ldcg(p.q + row_of(t) + other);
                    ko[t] = __ldcg(p.k + row_of(t) + other);
                    c[t] = __ldg(l.turn.cos_t + row);
                    s[t] = __ldg(l.turn.sin_t + row);
                }
#pragma unroll
                for (int t = 0; t < kGroup; ++t) {
                    if (!turns) continue;
                    q[t] = is_low ? rotated_low(q[t], qo[t], c[t], s[t]) : rotated_high(qo[t], q[t], c[t], s[t]);
                    k[t] = is_low ? rotated_low(k[t], ko[t], c[t], s[t]) : rotated_high(ko[t], k[t], c[t], s[t]);
                }
            }
            if (ranked) {
                const float bias = real ? __ldg(l.dt_bias + h * l.dim + d) : 0.0f;
#pragma unroll
                for (int t = 0; t < kGroup; ++t) g[t] = bias;
                const __nv_bfloat16* w = l.a2 + static_cast<size_t>(h * l.dim + (real ? d : 0u)) * l.a2_ld;      // a2_ld is the rank rounded up to 8 as well
                for (uint32_t c0 = 0; c0 < low_ld; c0 += 32) {
                    uint4 w8[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) w8[i] = c0 + 8 * i < low_ld ? __ldg(reinterpret_cast<const uint4*>(w + c0 + 8 * i)) : make_uint4(0, 0, 0, 0);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (c0 + 8 * i >= low_ld) break;
#pragma unroll
                        for (int t = 0; t < kGroup; ++t) {
                            const float4* x4 = reinterpret_cast<const float4*>(low + t * low_ld + c0 + 8 * i);
                            const float4 x0 = x4[0], x1 = x4[1];
                            const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
                            dense_fma8(w8[i], x, g[t]);
                        }
                    }
                }
            }
#pragma unroll
            for (int t = 0; t < kGroup; ++t) {
                const bool on = t0 + t < p.tokens;
                g[t] = !on ? 1.0f : ranked ? channel_decay(g[t], l.inv_tau) : fixed;
                q[t] = on && real ? q_scale * q[t] : 0.0f;
                k[t] = on && real ? k[t] : 0.0f;
            }
        } else {
#pragma unroll
            for (int t = 0; t < kGroup; ++t) {
                const bool on = t0 + t < p.tokens;
                g[t] = on ? __ldcg(p.g + (static_cast<size_t>(t0 + t) * p.heads + h) * kPitch + d) : 1.0f;
                q[t] = on ? __ldcg(p.q + (static_cast<size_t>(t0 + t) * p.q_heads + qh) * kPitch + d) : 0.0f;
                k[t] = !kDelta ? 1.0f - g[t] : on ? __ldcg(p.k + (static_cast<size_t>(t0 + t) * p.q_heads + qh) * kPitch + d) : 0.0f;
            }
        }
        float run = 1.0f;
#pragma unroll
        for (int t = 0; t < kGroup; ++t) {
            run *= g[t];
            if (kDelta) rec[t * kPitch + d] = k[t] * run;
            q_out[t * kPitch + d] = q[t] * run;
        }
        g_out[d] = run;
#pragma unroll
        for (int s = 0; s < kGroup; ++s) {
            float w = k[s];
            acc[28 + s * (s + 1) / 2 + s] = fmaf(q[s], w, acc[28 + s * (s + 1) / 2 + s]);
#pragma unroll
            for (int t = s + 1; t < kGroup; ++t) {
                w *= g[t];
                if (kDelta) acc[t * (t - 1) / 2 + s] = fmaf(k[t], w, acc[t * (t - 1) / 2 + s]);
                acc[28 + t * (t + 1) / 2 + s] = fmaf(q[t], w, acc[28 + t * (t + 1) / 2 + s]);
            }
            k_out[s * kPitch + d] = w;
        }
    }
    warp_sum64(acc, lane);
    sums[warp][2 * lane] = acc[0];
    sums[warp][2 * lane + 1] = acc[1];
    __syncwarp();
    float* const m_out = g_out + kPitch + (kDelta ? 64 : 0);
    if (kDelta) {
        if (lane < kGroup) {                                    // column `lane` of T by forward substitution
            float column[kGroup];
#pragma unroll
            for (int t = 0; t < kGroup; ++t) {
                float r = static_cast<int>(lane) == t ? 1.0f : 0.0f;
#pragma unroll
                for (int s = 0; s < t; ++s) r = fmaf(-sums[warp][t * (t - 1) / 2 + s], column[s], r);
                column[t] = t0 + t < p.tokens ? r * __ldcg(p.beta + static_cast<size_t>(t0 + t) * p.heads + h) : 0.0f;
                t_matrix[warp][t * 8 + lane] = column[t];
                g_out[kPitch + t * 8 + lane] = column[t];
            }
        }
        __syncwarp();
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {                               // two entries of M per lane
        const int t = (lane * 2 + e) / 8, c = (lane * 2 + e) % 8;
        float m = 0.0f;
        if (kDelta) {
            for (int s = c; s <= t; ++s) m = fmaf(sums[warp][28 + t * (t + 1) / 2 + s], t_matrix[warp][s * 8 + c], m);
        } else if (c <= t) {
            m = sums[warp][28 + t * (t + 1) / 2 + c];
        }
        m_out[t * 8 + c] = m;
    }
}

__device__ __forceinline__ void cp_async_4(float* smem_dst, const float* gmem_src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ uint64_t pf_add(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// sums[t][c] (8 tokens x 4 pairs of columns, partial per lane) -> the warp's sum of token lane / 4, pair lane % 4.
__device__ __forceinline__ uint64_t warp_sum_pairs(uint64_t (&v)[kGroup][4], uint32_t lane) {
    auto exchange = [](uint64_t keep, uint64_t give, int o) { return pf_add(keep, __shfl_xor_sync(0xffffffffu, give, o)); };
#pragma unroll
    for (int o = 16, n = 4; n >= 1; o >>= 1, n >>= 1) {         // lane bits 4, 3, 2: the token's bits
        const bool hi = lane & o;
#pragma unroll
        for (int t = 0; t < n; ++t)
#pragma unroll
            for (int c = 0; c < 4; ++c) v[t][c] = exchange(hi ? v[t + n][c] : v[t][c], hi ? v[t][c] : v[t + n][c], o);
    }
    const bool b1 = lane & 2, b0 = lane & 1;
    const uint64_t x = exchange(b1 ? v[0][2] : v[0][0], b1 ? v[0][0] : v[0][2], 2), y = exchange(b1 ? v[0][3] : v[0][1], b1 ? v[0][1] : v[0][3], 2);
    return exchange(b0 ? y : x, b0 ? x : y, 1);
}

// A CTA takes 32 columns of one head's state (its value channels), a warp eight of them.  A lane holds channels lane, lane + 32, ...
// of all eight columns, as four packed pairs of columns per channel, so a word of the record read from shared memory serves eight
// multiply-adds and every lane of the warp reads a different one.  kQuads = pitch / 32.  Grid: (ceil(vdim / 32), heads).
template <int kQuads, bool kDelta>
__global__ void __launch_bounds__(kScanThreads) state_scan_kernel(const __grid_constant__ ScanParams p) {
    constexpr uint32_t kPitch = kQuads * 32, kRecord = scan_record_floats(kPitch, kDelta), kStage = kRecord + kGroup * kScanColumns;
    constexpr uint32_t kQ = kDelta ? 8 * kPitch : 0, kK = kQ + 8 * kPitch, kG = kK + 8 * kPitch, kT = kG + kPitch, kM = kT + (kDelta ? 64 : 0);
    extern __shared__ __align__(16) float scan_smem[];
    pdl_launch_dependents();
    const uint32_t h = blockIdx.y, col_base = blockIdx.x * kScanColumns, groups = (p.tokens + kGroup - 1) / kGroup;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c0 = col_base + warp * 8;
    float* const u_rows = scan_smem + kScanStages * kStage + warp * kGroup * 8;      // this warp's u, [token][column]
    pdl_wait();
    auto stage = [&](uint32_t group) {
        float* dst = scan_smem + (group % kScanStages) * kStage;
        const float* rec = p.records + (static_cast<size_t>(group) * p.heads + h) * kRecord;
#pragma unroll 4
        for (uint32_t i = threadIdx.x; i < kRecord / 4; i += kScanThreads) cp_async_16(dst + i * 4, rec + i * 4, 16);
#pragma unroll
        for (uint32_t i = threadIdx.x; i < kGroup * kScanColumns; i += kScanThreads) {
            const uint32_t t = group * kGroup + i / kScanColumns, c = col_base + i % kScanColumns;
            float* d = dst + kRecord + i;
            if (c < p.vdim && t < p.tokens) cp_async_4(d, p.v + static_cast<size_t>(t) * p.v_ld + h * p.vdim + c); else *d = 0.0f;
        }
    };
    for (uint32_t i = 0; i < kScanStages - 1; ++i) {
        if (i < groups) stage(i);
        cp_async_commit();
    }
    uint64_t s[kQuads][4];
#pragma unroll
    for (int j = 0; j < kQuads; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const float* src = p.state + (static_cast<size_t>(h) * p.vdim + c0 + 2 * c) * kPitch + lane + 32 * j;
            s[j][c] = pf_pack(c0 + 2 * c < p.vdim ? __ldcg(src) : 0.0f, c0 + 2 * c + 1 < p.vdim ? __ldcg(src + kPitch) : 0.0f);
        }
    const uint32_t my_t = lane >> 2, my_pair = lane & 3;
    for (uint32_t group = 0; group < groups; ++group) {
        cp_async_wait<kScanStages - 2>();           // this group's copies have landed (this thread's; the barrier covers the others')
        __syncthreads();                            // ... and everybody is done with the buffer filled next
        if (group + kScanStages - 1 < groups) stage(group + kScanStages - 1);
        cp_async_commit();
        const float* rec = scan_smem + (group % kScanStages) * kStage;
        const float* v = rec + kRecord + warp * 8;
        const uint64_t zero2 = pf_pack(0.0f, 0.0f);
        auto with_state = [&](const float* rows) {  // rows [8][pitch] . S for this lane's token and pair of columns
            uint64_t sum[kGroup][4];
#pragma unroll
            for (int t = 0; t < kGroup; ++t)
#pragma unroll
                for (int j = 0; j < kQuads; ++j) {
                    const float w = rows[t * kPitch + lane + 32 * j];
                    const uint64_t ww = pf_pack(w, w);
#pragma unroll
                    for (int c = 0; c < 4; ++c) sum[t][c] = pf_fma(ww, s[j][c], j ? sum[t][c] : zero2);
                }
            return warp_sum_pairs(sum, lane);
        };
        const float2 v_mine = *reinterpret_cast<const float2*>(v + my_t * kScanColumns + my_pair * 2);
        uint64_t w_mine = pf_pack(v_mine.x, v_mine.y);
        if (kDelta) w_mine = pf_fma(with_state(rec), pf_pack(-1.0f, -1.0f), w_mine);
        uint64_t o = with_state(rec + kQ), u = zero2;
        // this lane's rows of T and M times the w of all eight tokens (columns of this lane's pair)
#pragma unroll
        for (int t4 = 0; t4 < 2; ++t4) {
            const float4 m4 = *reinterpret_cast<const float4*>(rec + kM + my_t * 8 + t4 * 4);
            const float4 x4 = kDelta ? *reinterpret_cast<const float4*>(rec + kT + my_t * 8 + t4 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float m[4] = {m4.x, m4.y, m4.z, m4.w}, x[4] = {x4.x, x4.y, x4.z, x4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint64_t w = __shfl_sync(0xffffffffu, w_mine, (t4 * 4 + i) * 4 + static_cast<int>(my_pair));
                o = pf_fma(pf_pack(m[i], m[i]), w, o);
                if (kDelta) u = pf_fma(pf_pack(x[i], x[i]), w, u);
            }
        }
        const uint32_t t_mine = group * kGroup + my_t, c_mine = c0 + my_pair * 2;
        if (t_mine < p.tokens) {
            float o0, o1;
            pf_unpack(o, o0, o1);
            float* dst = p.out + (static_cast<size_t>(t_mine) * p.heads + h) * p.vdim + c_mine;
            if (c_mine < p.vdim) dst[0] = o0;
            if (c_mine + 1 < p.vdim) dst[1] = o1;
        }
        const float* u_src = v;
        uint32_t u_ld = kScanColumns;
        if (kDelta) {
            *reinterpret_cast<uint64_t*>(u_rows + my_t * 8 + my_pair * 2) = u;
            __syncwarp();
            u_src = u_rows;
            u_ld = 8;
        }
#pragma unroll
        for (int j = 0; j < kQuads; ++j) {
            const float g = rec[kG + lane + 32 * j];
            const uint64_t gg = pf_pack(g, g);
#pragma unroll
            for (int c = 0; c < 4; ++c) s[j][c] = pf_mul(s[j][c], gg);
        }
#pragma unroll
        for (int t = 0; t < kGroup; ++t) {
            const float4 ua = *reinterpret_cast<const float4*>(u_src + t * u_ld), ub = *reinterpret_cast<const float4*>(u_src + t * u_ld + 4);
            const uint64_t uu[4] = {pf_pack(ua.x, ua.y), pf_pack(ua.z, ua.w), pf_pack(ub.x, ub.y), pf_pack(ub.z, ub.w)};
#pragma unroll
            for (int j = 0; j < kQuads; ++j) {
                const float k = rec[kK + t * kPitch + lane + 32 * j];
                const uint64_t kk = pf_pack(k, k);
#pragma unroll
                for (int c = 0; c < 4; ++c) s[j][c] = pf_fma(kk, uu[c], s[j][c]);
            }
        }
        if (kDelta) __syncwarp();                   // u_rows is read before the next group writes it
    }
#pragma unroll
    for (int j = 0; j < kQuads; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            float* dst = p.state + (static_cast<size_t>(h) * p.vdim + c0 + 2 * c) * kPitch + lane + 32 * j;
            float a, b;
            pf_unpack(s[j][c], a, b);
            if (c0 + 2 * c < p.vdim) dst[0] = a;
            if (c0 + 2 * c + 1 < p.vdim) dst[kPitch] = b;
        }
}

// ---- one token -------------------------------------------------------------------------------------------------------

// One CTA per head: everything from the projections of one token to the output projection's input.  proj: delta rule
// q | k | v | b | a1 | g1, gated write q | f | v, decayed write q | k | v | g | a1 (a1 without constant decays).  out [heads][vdim].
// kMaxQuads: most 16-byte words a lane holds of a column (pitch / 32): up to four, a CTA of 1024 threads takes 128 columns at a time.
__host__ __device__ constexpr int step_threads(int max_quads) { return max_quads <= 4 ? 1024 : 512; }
__host__ __device__ inline uint32_t step_low_floats(const LinearLayer& l) { return ((l.rank_a + 63) & ~63u) + ((l.rank_g + 63) & ~63u); }
template <int kRule, int kMaxQuads>
__global__ void __launch_bounds__(step_threads(kMaxQuads)) state_step_kernel(const __grid_constant__ LinearLayer l, const float* __restrict__ proj,
                                                                  const int* __restrict__ pos_ptr, float* __restrict__ out) {
    constexpr bool kDelta = kRule == kDeltaRule;
    constexpr uint32_t kStepThreads = step_threads(kMaxQuads), kWarps = kStepThreads / 32;
    extern __shared__ __align__(16) float low[];                   // a1 and (delta rule) g1 outputs, each padded with zeros to 64
    __shared__ __align__(16) float q[256], k[256], g[256];
    __shared__ float v[256], o[256], gate[256], bias[256], norm[256];
    const uint32_t h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane & 7, quads = l.pitch / 32;
    pdl_launch_dependents();
    // rows of the rank projections, eight lanes to a row (decays first, then the gate): weights, so their first kAhead words per
    // lane are fetched while the previous launch is still running
    constexpr uint32_t kAhead = kMaxQuads <= 4 ? 4 : 8;
    uint4 ahead[kAhead];
    const bool ranked = kDelta || (kRule == kDecayedWrite && !l.decay);
    const uint32_t words = ranked ? (max(l.a2_ld, l.g2_ld) + 63) / 64 : 0;      // 16-byte words per lane and row
    uint32_t rank_rows = ranked ? l.pitch : 0;
    if (kDelta) rank_rows += l.vdim;
    auto rank_row = [&](uint32_t r, uint32_t& ld) -> const __nv_bfloat16* {     // null: padding
        const bool is_g = r >= l.pitch;
        const uint32_t d = is_g ? r - l.pitch : r;
        ld = is_g ? l.g2_ld : l.a2_ld;
        if (r >= rank_rows || d >= (is_g ? l.vdim : l.dim)) return nullptr;
        return is_g ? l.g2 + static_cast<size_t>(h * l.vdim + d) * ld : l.a2 + static_cast<size_t>(h * l.dim + d) * ld;
    };
    if (ranked) {
        uint32_t r = warp * 4 + (lane >> 3), word = 0;
#pragma unroll
        for (uint32_t i = 0; i < kAhead; ++i) {
            uint32_t ld = 0;
            const __nv_bfloat16* w = rank_row(r, ld);
            const uint32_t c = (word * 8 + part) * 8;
            ahead[i] = w && c < ld ? __ldg(reinterpret_cast<const uint4*>(w + c)) : make_uint4(0, 0, 0, 0);
            if (++word == words) { word = 0; r += kWarps * 4; }
        }
    }
    // so are the small constants that would otherwise cost a round trip each in the middle of the step
    for (uint32_t i = threadIdx.x; i < l.vdim; i += kStepThreads) norm[i] = __ldg(l.norm + i);
    if (ranked)
        for (uint32_t i = threadIdx.x; i < l.dim; i += kStepThreads) bias[i] = __ldg(l.dt_bias + h * l.dim + i);
    const float a_scale = kDelta ? -expf(__ldg(l.a_log + h)) : 0.0f, fixed = kRule == kDecayedWrite && l.decay ? __ldg(l.decay + h) : 0.0f;
    pdl_wait();
    // the first columns' state words are on their way while the token's vectors are formed
    float* const state = l.state + static_cast<size_t>(h) * l.vdim * l.pitch + part * 4;
    uint32_t col = warp * 4 + (lane >> 3);
    float4 pre[kMaxQuads];
#pragma unroll
    for (uint32_t i = 0; i < kMaxQuads; ++i)
        pre[i] = (i < quads && col < l.vdim) ? __ldcg(reinterpret_cast<const float4*>(state + static_cast<size_t>(col) * l.pitch + i * 32)) : make_float4(0.f, 0.f, 0.f, 0.f);
    float beta = 0.0f;
    // the decays, and the delta rule's output gate, from the low-rank inputs
    const uint32_t pad_a = (l.rank_a + 63) & ~63u;
    auto stage_low = [&](const float* a1, const float* g1) {
        for (uint32_t i = threadIdx.x; i < step_low_floats(l); i += kStepThreads) {
            const bool is_g = i >= pad_a;
            const uint32_t c = is_g ? i - pad_a : i;
            low[i] = c < (is_g ? l.rank_g : l.rank_a) ? __ldcg((is_g ? g1 : a1) + c) : 0.0f;
        }
    };
    auto low_rank = [&] {
        uint32_t r = warp * 4 + (lane >> 3), word = 0;
        float acc = 0.0f;
        auto take = [&](const uint4& w) {
            const bool is_g = r >= l.pitch;
            const uint32_t c = (word * 8 + part) * 8;
            if (c < (is_g ? l.g2_ld : l.a2_ld)) {
                const float4* in = reinterpret_cast<const float4*>(low + (is_g ? pad_a : 0u) + c);
                const float4 x0 = in[0], x1 = in[1];
                const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
                dense_fma8(w, x, acc);
            }
            ++word;
            if (word != words) return;
#pragma unroll
            for (int s = 1; s < 8; s <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, s);
            if (part == 0 && r < rank_rows) {
                if (is_g) gate[r - l.pitch] = logistic(acc);
                else if (kDelta) g[r] = r < l.dim ? expf(a_scale * softplus_f(acc + bias[r])) : 0.0f;
                else g[r] = r < l.dim ? channel_decay(acc + bias[r], l.inv_tau) : 0.0f;
            }
            acc = 0.0f;
            word = 0;
            r += kWarps * 4;
        };
        // r - lane / 8 and word are the same in all lanes of a warp, so the loops below do not diverge around the shuffles
#pragma unroll
        for (uint32_t i = 0; i < kAhead; ++i)
            if (r - (lane >> 3) < rank_rows) take(ahead[i]);
        while (r - (lane >> 3) < rank_rows) {
            uint32_t ld = 0;
            const __nv_bfloat16* w = rank_row(r, ld);
            const uint32_t c = (word * 8 + part) * 8;
            take(w && c < ld ? __ldg(reinterpret_cast<const uint4*>(w + c)) : make_uint4(0, 0, 0, 0));
        }
    };
    if (kDelta) {
        const int pos = *pos_ptr;
        const uint32_t channels = linear_channels(l), kd = l.kv_heads * l.dim, qh = h / (l.heads / l.kv_heads);
        stage_low(proj + channels + l.heads, proj + channels + l.heads + l.rank_a);
        beta = logistic(__ldcg(proj + channels + h));
        const bool owner = h % (l.heads / l.kv_heads) == 0;        // one CTA per q/k head keeps its ring
        float* slot = l.conv.ring + static_cast<size_t>(static_cast<uint32_t>(pos) % l.conv.taps) * channels;
        for (uint32_t i = threadIdx.x; i < 2 * l.pitch + l.vdim; i += kStepThreads) {
            const bool is_v = i >= 2 * l.pitch, is_k = !is_v && i >= l.pitch;
            const uint32_t d = is_v ? i - 2 * l.pitch : is_k ? i - l.pitch : i;
            float y = 0.0f;
            if (is_v || d < l.dim) {
                const uint32_t c = is_v ? 2 * kd + h * l.vdim + d : (is_k ? kd : 0u) + qh * l.dim + d;
                y = silu_f(conv_sum(l.conv, proj + c, 0, 0, pos, c));
                if (is_v || owner) slot[c] = __ldcg(proj + c);
            }
            (is_v ? v : is_k ? k : q)[d] = y;
        }
        __syncthreads();
        low_rank();
        __syncthreads();
        if (warp < 2) {                                            // unit norms: warp 0 takes q, warp 1 k
            float* x = warp ? k : q;
            float ss = 0.0f;
            for (uint32_t d = lane; d < l.pitch; d += 32) ss += x[d] * x[d];
            float inv = 1.0f / sqrtf(warp_sum(ss) + kUnitEps);
            if (!warp) inv *= 1.0f / sqrtf(static_cast<float>(l.dim));
            for (uint32_t d = lane; d < l.pitch; d += 32) x[d] *= inv;
        }
    } else if (kRule == kDecayedWrite) {
        const uint32_t kd = l.heads * l.dim, nv = l.heads * l.vdim;
        const size_t row = l.turn.half ? rotation_row(l.turn, *pos_ptr) : 0;
        const float q_scale = 1.0f / sqrtf(static_cast<float>(l.dim));
        if (ranked) stage_low(proj + 2 * kd + 2 * nv, nullptr);
        for (uint32_t i = threadIdx.x; i < 2 * (l.pitch + l.vdim); i += kStepThreads) {
            if (i < 2 * l.pitch) {
                const bool is_k = i >= l.pitch;
                const uint32_t d = is_k ? i - l.pitch : i;
                const float* x = proj + (is_k ? kd : 0u) + h * l.dim;
                const float y = d < l.dim ? rotated(l.turn, [&](uint32_t j) { return __ldcg(x + j); }, d, row) : 0.0f;
                if (is_k) k[d] = y; else q[d] = y * q_scale;
                if (!ranked && !is_k) g[d] = fixed;
            } else {
                const bool is_g = i >= 2 * l.pitch + l.vdim;
                const uint32_t d = i - 2 * l.pitch - (is_g ? l.vdim : 0u);
                const float y = __ldcg(proj + 2 * kd + (is_g ? nv : 0u) + h * l.vdim + d);
                if (is_g) gate[d] = silu_f(y); else v[d] = y;
            }
        }
        if (ranked) {
            __syncthreads();
            low_rank();
        }
    } else {
        for (uint32_t d = threadIdx.x; d < l.pitch; d += kStepThreads) {
            const uint32_t c = h * l.dim + d;
            float qv = 0.0f, fv = 1.0f;
            if (d < l.dim) {
                qv = silu_f(__ldcg(proj + c));
                fv = l.lower[c] + (1.0f - l.lower[c]) * logistic(__ldcg(proj + l.heads * l.dim + c) + l.f_bias[c]);
            }
            q[d] = qv;
            g[d] = fv;
            k[d] = 1.0f - fv;
        }
        for (uint32_t i = threadIdx.x; i < l.vdim; i += kStepThreads) v[i] = __ldcg(proj + 2 * l.heads * l.dim + h * l.vdim + i);
    }
    __syncthreads();
    // a warp takes four columns at a time, eight lanes to a column
    for (uint32_t base = warp * 4; base < l.vdim; base += kWarps * 4) {
        col = base + (lane >> 3);
        const bool on = col < l.vdim;
        float* mine = state + static_cast<size_t>(col) * l.pitch;
        float4 s[kMaxQuads];
        float u = on ? v[col] : 0.0f, dot = 0.0f;
#pragma unroll
        for (uint32_t i = 0; i < kMaxQuads; ++i) {
            if (i >= quads) break;
            s[i] = base == warp * 4 ? pre[i] : on ? __ldcg(reinterpret_cast<const float4*>(mine + i * 32)) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 gg = reinterpret_cast<const float4*>(g)[i * 8 + part], kk = reinterpret_cast<const float4*>(k)[i * 8 + part];
            s[i] = make_float4(s[i].x * gg.x, s[i].y * gg.y, s[i].z * gg.z, s[i].w * gg.w);
            if (kDelta) dot += s[i].x * kk.x + s[i].y * kk.y + s[i].z * kk.z + s[i].w * kk.w;
        }
        if (kDelta) {
#pragma unroll
            for (int b = 1; b < 8; b <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, b);
            u = beta * (u - dot);
        }
        float acc = 0.0f;
#pragma unroll
        for (uint32_t i = 0; i < kMaxQuads; ++i) {
            if (i >= quads) break;
            const float4 qq = reinterpret_cast<const float4*>(q)[i * 8 + part], kk = reinterpret_cast<const float4*>(k)[i * 8 + part];
            s[i] = make_float4(fmaf(kk.x, u, s[i].x), fmaf(kk.y, u, s[i].y), fmaf(kk.z, u, s[i].z), fmaf(kk.w, u, s[i].w));
            acc += s[i].x * qq.x + s[i].y * qq.y + s[i].z * qq.z + s[i].w * qq.w;
            if (on) *reinterpret_cast<float4*>(mine + i * 32) = s[i];
        }
#pragma unroll
        for (int b = 1; b < 8; b <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, b);
        if (on && part == 0) o[col] = acc;
    }
    __syncthreads();
    float ss = 0.0f;
    for (uint32_t i = lane; i < l.vdim; i += 32) ss += o[i] * o[i];          // every warp forms the head's norm itself
    const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(l.vdim) + l.eps);
    for (uint32_t i = threadIdx.x; i < l.vdim; i += kStepThreads) out[h * l.vdim + i] = o[i] * inv * norm[i] * (kRule == kGatedWrite ? 1.0f : gate[i]);
}

}  // namespace zk
