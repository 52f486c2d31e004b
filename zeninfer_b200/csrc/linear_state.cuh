// Mixers with a matrix state per head, S [dim][vdim] in fp32, carried from token to token:
//
//   delta rule    S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (g per key channel)
//   gated write   S <- f * S + (1 - f) v^T;           o = S^T q                       (f per key channel, no key)
//
// state_scan_kernel walks a block of tokens with the state in registers, state_step_kernel takes one token and does everything
// between the layer's input projections and its output projection.  The kernels around the scan form its inputs (short causal
// convolution, unit norms, decays, gates) for all tokens at once.
//
// Device layout of a state: [heads][vdim][pitch], pitch = dim rounded up to 32 and zero beyond dim, so that eight lanes read a
// column's rows as consecutive 16-byte words.  The convolution keeps the inputs of the last `taps` tokens in a ring
// [taps][channels] whose slot is the position modulo taps: a token reads the taps - 1 slots before its own and nobody else
// writes those, so it needs no second buffer.
#pragma once
#include "gemv_bf16.cuh"

namespace zk {

__device__ __forceinline__ float silu_f(float z) { return z * logistic(z); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z + log1pf(expf(-z)) : log1pf(expf(z)); }
constexpr float kUnitEps = 1e-6f;

struct LinearLayer {
    uint32_t heads, kv_heads, dim, vdim, pitch;
    uint32_t taps;                 // delta rule: convolution taps
    uint32_t rank_a, rank_g;       // delta rule: ranks of the decay's and the output gate's projections
    uint32_t a2_ld, g2_ld;
    const float* conv;             // [taps][channels]: q, k, v channels
    const float* a_log;            // [heads]
    const float* dt_bias;          // [heads][dim]
    const __nv_bfloat16* a2;       // [heads dim][a2_ld]
    const __nv_bfloat16* g2;       // [heads vdim][g2_ld]
    const float* f_bias;           // gated write: [heads][dim]
    const float* lower;            // gated write: [heads][dim]
    const float* norm;             // [vdim]
    float* ring;                   // [taps][channels]
    float* state;                  // [heads][vdim][pitch]
    float eps;
};
__host__ __device__ inline uint32_t linear_channels(const LinearLayer& l) { return 2 * l.kv_heads * l.dim + l.heads * l.vdim; }

// Convolution of channel c at block row t (position pos + t), then silu.  x: projection rows of pitch ld, channel c at column c;
// rows before the block come from the ring, tokens before the sequence's start are zeros.
__device__ __forceinline__ float conv_silu(const LinearLayer& l, const float* __restrict__ x, uint32_t ld, int t, int pos, uint32_t c, uint32_t channels) {
    float y = 0.0f;
    const int taps = static_cast<int>(l.taps);
#pragma unroll 4
    for (int j = 0; j < taps; ++j) {
        const int s = t - (taps - 1 - j), at = pos + s;
        const float* src = s >= 0 ? x + static_cast<size_t>(s) * ld + c : l.ring + static_cast<size_t>(static_cast<uint32_t>(max(at, 0)) % l.taps) * channels + c;
        const float v = at >= 0 ? __ldcg(src) : 0.0f;
        y = fmaf(__ldg(l.conv + static_cast<size_t>(j) * channels + c), v, y);
    }
    return silu_f(y);
}

// ---- inputs of the scan for a block of tokens -------------------------------------------------------------------------

constexpr int kStrip = 8;          // tokens a warp takes at a time: a channel's inputs stay in registers while the taps slide over them
constexpr int kMaxSlidingTaps = 8; // more taps than this are read again for every token

// y[i] = silu(convolution) of channel c at tokens t0 .. t0 + n - 1 (n <= kStrip; the rest is not used).
__device__ __forceinline__ void conv_silu_strip(const LinearLayer& l, const float* __restrict__ x, uint32_t ld, int t0, int n, int pos, uint32_t c,
                                                uint32_t channels, float (&y)[kStrip]) {
    const int taps = static_cast<int>(l.taps);
    if (taps > kMaxSlidingTaps) {
#pragma unroll
        for (int i = 0; i < kStrip; ++i)
            if (i < n) y[i] = conv_silu(l, x, ld, t0 + i, pos, c, channels);
        return;
    }
    float w[kMaxSlidingTaps], in[kMaxSlidingTaps - 1 + kStrip];       // w right-aligned: w[7] is the current token's; in[7 + i]: token t0 + i
#pragma unroll
    for (int j = 0; j < kMaxSlidingTaps; ++j) {
        const int tap = j - (kMaxSlidingTaps - taps);
        w[j] = tap >= 0 ? __ldg(l.conv + static_cast<size_t>(tap) * channels + c) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < kMaxSlidingTaps - 1 + kStrip; ++i) {
        const int s = t0 + i - (kMaxSlidingTaps - 1), at = pos + s;   // block row, position
        in[i] = 0.0f;
        if (at >= 0 && s >= t0 - (taps - 1) && s < t0 + n)
            in[i] = s >= 0 ? __ldcg(x + static_cast<size_t>(s) * ld + c) : l.ring[static_cast<size_t>(static_cast<uint32_t>(at) % l.taps) * channels + c];
    }
#pragma unroll
    for (int i = 0; i < kStrip; ++i) {
        float sum = 0.0f;
#pragma unroll
        for (int j = 0; j < kMaxSlidingTaps; ++j) sum = fmaf(w[j], in[i + j], sum);
        y[i] = silu_f(sum);
    }
}

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
    const uint32_t qk_items = 2 * l.kv_heads, v_items = (nv + 31) / 32, items = qk_items + v_items + l.heads;
    for (uint32_t item = blockIdx.y * 8 + (threadIdx.x >> 5); item < items; item += gridDim.y * 8) {
        float y[kStrip];
        if (item < qk_items) {
            const bool is_q = item < l.kv_heads;
            const uint32_t head = is_q ? item : item - l.kv_heads, c0 = (is_q ? 0u : kd) + head * l.dim;
            float* dst = (is_q ? q : k) + (static_cast<size_t>(t0) * l.kv_heads + head) * l.pitch;
            const float scale = is_q ? 1.0f / sqrtf(static_cast<float>(l.dim)) : 1.0f;
            float ss[kStrip];
#pragma unroll
            for (int i = 0; i < kStrip; ++i) ss[i] = 0.0f;
            for (uint32_t d = lane; d < l.pitch; d += 32) {            // unscaled first: a lane reads back only what it wrote
#pragma unroll
                for (int i = 0; i < kStrip; ++i) y[i] = 0.0f;
                if (d < l.dim) conv_silu_strip(l, proj, ld, t0, n, pos, c0 + d, channels, y);
#pragma unroll
                for (int i = 0; i < kStrip; ++i)
                    if (i < n) { ss[i] += y[i] * y[i]; dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + d] = y[i]; }
            }
#pragma unroll
            for (int i = 0; i < kStrip; ++i) ss[i] = scale / sqrtf(warp_sum(ss[i]) + kUnitEps);
            for (uint32_t d = lane; d < l.pitch; d += 32) {
#pragma unroll
                for (int i = 0; i < kStrip; ++i)
                    if (i < n) dst[static_cast<size_t>(i) * l.kv_heads * l.pitch + d] *= ss[i];
            }
        } else if (item < qk_items + v_items) {
            const uint32_t c = (item - qk_items) * 32 + lane;
            if (c >= nv) continue;
            conv_silu_strip(l, proj, ld, t0, n, pos, 2 * kd + c, channels, y);
#pragma unroll
            for (int i = 0; i < kStrip; ++i)
                if (i < n) v[static_cast<size_t>(t0 + i) * nv + c] = y[i];
        } else {
            const uint32_t h = item - qk_items - v_items;
            const float rate = -expf(l.a_log[h]);
            for (uint32_t d = lane; d < l.pitch; d += 32) {
                const float bias = d < l.dim ? l.dt_bias[h * l.dim + d] : 0.0f;
#pragma unroll
                for (int i = 0; i < kStrip; ++i)
                    if (i < n)
                        g[(static_cast<size_t>(t0 + i) * l.heads + h) * l.pitch + d] =
                            d < l.dim ? expf(rate * softplus_f(__ldcg(decay + static_cast<size_t>(t0 + i) * decay_ld + h * l.dim + d) + bias)) : 0.0f;
            }
            if (static_cast<int>(lane) < n) beta[static_cast<size_t>(t0 + lane) * l.heads + h] = logistic(__ldcg(proj + static_cast<size_t>(t0 + lane) * ld + channels + h));
        }
    }
}

// The ring after a block of T tokens: the inputs of its last min(T, taps) tokens.  Runs after the kernel above.
__global__ void __launch_bounds__(256) conv_ring_update_kernel(const __grid_constant__ LinearLayer l, const float* __restrict__ proj, uint32_t ld, uint32_t tokens,
                                                               const int* __restrict__ pos_ptr) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t channels = linear_channels(l), c = blockIdx.x * 256 + threadIdx.x, pos = static_cast<uint32_t>(*pos_ptr);
    if (c >= channels) return;
    for (uint32_t t = tokens > l.taps ? tokens - l.taps : 0; t < tokens; ++t)
        l.ring[static_cast<size_t>((pos + t) % l.taps) * channels + c] = proj[static_cast<size_t>(t) * ld + c];
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

struct ScanParams {
    const float* q;        // [T][q_heads][pitch]
    const float* k;        // [T][q_heads][pitch]; delta rule only
    const float* g;        // [T][heads][pitch]
    const float* v;        // [T][v_ld], head h's values at column h * vdim
    const float* beta;     // [T][heads]; delta rule only
    float* state;          // [heads][vdim][pitch]
    float* out;            // [T][heads][vdim]
    uint32_t tokens, heads, q_heads, vdim, v_ld;
};

constexpr int kScanThreads = 128, kScanColumns = 32, kScanTokens = 8, kScanStages = 4;    // columns of S per CTA; tokens per staged block; blocks in flight
template <int kQuads, bool kDelta>
__host__ __device__ constexpr uint32_t scan_token_floats() { return (kDelta ? 3 : 2) * kQuads * 32 + kScanColumns + 4; }
template <int kQuads, bool kDelta>
__host__ __device__ constexpr uint32_t scan_smem_bytes() { return kScanStages * kScanTokens * scan_token_floats<kQuads, kDelta>() * 4; }

__device__ __forceinline__ void cp_async_4(float* smem_dst, const float* gmem_src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(gmem_src) : "memory");
}

// A CTA takes 32 columns of one head's state (its value channels), a warp eight of them.  A column's rows are spread over eight
// lanes, lane `part` holding the 16-byte words part, part + 8, ...; a lane holds two columns, so a word of q, k or g read from
// shared memory serves both.  The state never leaves the registers between the block's first and last token; arithmetic is packed
// fp32 pairs.  Tokens go in groups of eight: only the delta rule's own sum is reduced token by token (it is what the next token
// waits for); the read-outs of a group stay as partial sums and are reduced together, after which lane `part` holds token `part`'s.
// A group's missing tokens at the end of the block are staged as g = 1 and zeros: they leave the state as it is.
// kQuads = pitch / 32.  Grid: (ceil(vdim / 32), heads).
template <int kQuads, bool kDelta>
__global__ void __launch_bounds__(kScanThreads) state_scan_kernel(const __grid_constant__ ScanParams p) {
    constexpr uint32_t kPitch = kQuads * 32, kToken = scan_token_floats<kQuads, kDelta>();
    constexpr uint32_t kG = 0, kQ = kPitch, kK = 2 * kPitch, kV = (kDelta ? 3 : 2) * kPitch, kB = kV + kScanColumns;
    extern __shared__ __align__(16) float scan_smem[];
    pdl_launch_dependents();
    const uint32_t h = blockIdx.y, qh = h / (p.heads / p.q_heads), col_base = blockIdx.x * kScanColumns;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane & 7;
    const uint32_t local = warp * 8 + (lane >> 3) * 2, c0 = col_base + local;      // this lane's columns: c0, c0 + 1
    const bool on0 = c0 < p.vdim, on1 = c0 + 1 < p.vdim;
    pdl_wait();
    auto stage = [&](uint32_t t0, uint32_t buf) {
        float* dst = scan_smem + buf * kScanTokens * kToken;
        constexpr uint32_t kWords = kPitch / 4, kRows = kDelta ? 3 : 2;
#pragma unroll 4
        for (uint32_t i = threadIdx.x; i < kScanTokens * kRows * kWords; i += kScanThreads) {
            const uint32_t t = i / (kRows * kWords), rest = i % (kRows * kWords), row = rest / kWords, word = rest % kWords;
            float* d = dst + t * kToken + row * kPitch + word * 4;
            if (t0 + t < p.tokens) {
                const float* src = row == 0 ? p.g + (static_cast<size_t>(t0 + t) * p.heads + h) * kPitch
                                            : (row == 1 ? p.q : p.k) + (static_cast<size_t>(t0 + t) * p.q_heads + qh) * kPitch;
                cp_async_16(d, src + word * 4, 16);
            } else {
                const float fill = row == 0 ? 1.0f : 0.0f;
                *reinterpret_cast<float4*>(d) = make_float4(fill, fill, fill, fill);
            }
        }
#pragma unroll
        for (uint32_t i = threadIdx.x; i < kScanTokens * kScanColumns; i += kScanThreads) {
            const uint32_t t = i / kScanColumns, c = i % kScanColumns;
            float* d = dst + t * kToken + kV + c;
            if (col_base + c < p.vdim && t0 + t < p.tokens) cp_async_4(d, p.v + static_cast<size_t>(t0 + t) * p.v_ld + h * p.vdim + col_base + c); else *d = 0.0f;
        }
        if (kDelta && threadIdx.x < kScanTokens) {
            float* d = dst + threadIdx.x * kToken + kB;
            if (t0 + threadIdx.x < p.tokens) cp_async_4(d, p.beta + static_cast<size_t>(t0 + threadIdx.x) * p.heads + h); else *d = 0.0f;
        }
    };
    for (uint32_t i = 0; i < kScanStages - 1; ++i) {
        if (i * kScanTokens < p.tokens) stage(i * kScanTokens, i);
        cp_async_commit();
    }
    uint64_t s[2][kQuads][2];
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const float* src = p.state + (static_cast<size_t>(h) * p.vdim + c0 + c) * kPitch + part * 4;
#pragma unroll
        for (int i = 0; i < kQuads; ++i) {
            const float4 w = (c ? on1 : on0) ? __ldcg(reinterpret_cast<const float4*>(src + i * 32)) : make_float4(0.f, 0.f, 0.f, 0.f);
            s[c][i][0] = pf_pack(w.x, w.y);
            s[c][i][1] = pf_pack(w.z, w.w);
        }
    }
    const uint64_t zero2 = pf_pack(0.0f, 0.0f);
    uint32_t group = 0;
    for (uint32_t t0 = 0; t0 < p.tokens; t0 += kScanTokens, ++group) {
        cp_async_wait<kScanStages - 2>();           // this group's copies have landed (this thread's; the barrier covers the others')
        __syncthreads();                            // ... and everybody is done with the buffer filled next
        const uint32_t ahead = t0 + (kScanStages - 1) * kScanTokens;
        if (ahead < p.tokens) stage(ahead, (group + kScanStages - 1) % kScanStages);
        cp_async_commit();
        const float* tok = scan_smem + (group % kScanStages) * kScanTokens * kToken;
        float out[2][kScanTokens];
#pragma unroll
        for (int t = 0; t < kScanTokens; ++t, tok += kToken) {
            uint64_t g[kQuads][2], q[kQuads][2], k[kQuads][2];
#pragma unroll
            for (int i = 0; i < kQuads; ++i) {
                const float4 a = reinterpret_cast<const float4*>(tok + kG)[i * 8 + part], b = reinterpret_cast<const float4*>(tok + kQ)[i * 8 + part];
                g[i][0] = pf_pack(a.x, a.y); g[i][1] = pf_pack(a.z, a.w);
                q[i][0] = pf_pack(b.x, b.y); q[i][1] = pf_pack(b.z, b.w);
                if (kDelta) {
                    const float4 c = reinterpret_cast<const float4*>(tok + kK)[i * 8 + part];
                    k[i][0] = pf_pack(c.x, c.y); k[i][1] = pf_pack(c.z, c.w);
                } else {
                    k[i][0] = pf_pack(1.0f - a.x, 1.0f - a.y); k[i][1] = pf_pack(1.0f - a.z, 1.0f - a.w);
                }
            }
            const float2 v2 = *reinterpret_cast<const float2*>(tok + kV + local);
            float u[2] = {v2.x, v2.y};
            if (kDelta) {
                const float beta = tok[kB];
                float dot[2];
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    uint64_t d0 = zero2, d1 = zero2;
#pragma unroll
                    for (int i = 0; i < kQuads; ++i) {
                        s[c][i][0] = pf_mul(s[c][i][0], g[i][0]);
                        s[c][i][1] = pf_mul(s[c][i][1], g[i][1]);
                        d0 = pf_fma(s[c][i][0], k[i][0], d0);
                        d1 = pf_fma(s[c][i][1], k[i][1], d1);
                    }
                    float a, b, e, f;
                    pf_unpack(d0, a, b);
                    pf_unpack(d1, e, f);
                    dot[c] = (a + b) + (e + f);
                }
#pragma unroll
                for (int o = 1; o < 8; o <<= 1) {
                    dot[0] += __shfl_xor_sync(0xffffffffu, dot[0], o);
                    dot[1] += __shfl_xor_sync(0xffffffffu, dot[1], o);
                }
                u[0] = beta * (u[0] - dot[0]);
                u[1] = beta * (u[1] - dot[1]);
            }
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const uint64_t uu = pf_pack(u[c], u[c]);
                uint64_t d0 = zero2, d1 = zero2;
#pragma unroll
                for (int i = 0; i < kQuads; ++i) {
                    if (kDelta) {
                        s[c][i][0] = pf_fma(k[i][0], uu, s[c][i][0]);
                        s[c][i][1] = pf_fma(k[i][1], uu, s[c][i][1]);
                    } else {
                        s[c][i][0] = pf_fma(k[i][0], uu, pf_mul(s[c][i][0], g[i][0]));
                        s[c][i][1] = pf_fma(k[i][1], uu, pf_mul(s[c][i][1], g[i][1]));
                    }
                    d0 = pf_fma(s[c][i][0], q[i][0], d0);
                    d1 = pf_fma(s[c][i][1], q[i][1], d1);
                }
                float a, b, e, f;
                pf_unpack(d0, a, b);
                pf_unpack(d1, e, f);
                out[c][t] = (a + b) + (e + f);
            }
        }
        // eight partial read-outs per column over eight lanes: each exchange halves the tokens a lane carries
        const bool b2 = part & 4, b1 = part & 2, b0 = part & 1;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            float r4[4], r2[2];
#pragma unroll
            for (int i = 0; i < 4; ++i) r4[i] = (b2 ? out[c][i + 4] : out[c][i]) + __shfl_xor_sync(0xffffffffu, b2 ? out[c][i] : out[c][i + 4], 4);
#pragma unroll
            for (int i = 0; i < 2; ++i) r2[i] = (b1 ? r4[i + 2] : r4[i]) + __shfl_xor_sync(0xffffffffu, b1 ? r4[i] : r4[i + 2], 2);
            const float o = (b0 ? r2[1] : r2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? r2[0] : r2[1], 1);
            if ((c ? on1 : on0) && t0 + part < p.tokens) p.out[(static_cast<size_t>(t0 + part) * p.heads + h) * p.vdim + c0 + c] = o;
        }
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        float* dst = p.state + (static_cast<size_t>(h) * p.vdim + c0 + c) * kPitch + part * 4;
        if (!(c ? on1 : on0)) continue;
#pragma unroll
        for (int i = 0; i < kQuads; ++i) {
            float4 w;
            pf_unpack(s[c][i][0], w.x, w.y);
            pf_unpack(s[c][i][1], w.z, w.w);
            *reinterpret_cast<float4*>(dst + i * 32) = w;
        }
    }
}

// ---- one token -------------------------------------------------------------------------------------------------------

// One CTA per head: everything from the projections of one token to the output projection's input.  proj: delta rule
// q | k | v | b | a1 | g1, gated write q | f | v.  out [heads][vdim].
// kMaxQuads: most 16-byte words a lane holds of a column (pitch / 32): up to four, a CTA of 1024 threads takes 128 columns at a time.
__host__ __device__ constexpr int step_threads(int max_quads) { return max_quads <= 4 ? 1024 : 512; }
__host__ __device__ inline uint32_t step_low_floats(const LinearLayer& l) { return ((l.rank_a + 63) & ~63u) + ((l.rank_g + 63) & ~63u); }
template <bool kDelta, int kMaxQuads>
__global__ void __launch_bounds__(step_threads(kMaxQuads)) state_step_kernel(const __grid_constant__ LinearLayer l, const float* __restrict__ proj,
                                                                  const int* __restrict__ pos_ptr, float* __restrict__ out) {
    constexpr uint32_t kStepThreads = step_threads(kMaxQuads), kWarps = kStepThreads / 32;
    extern __shared__ __align__(16) float low[];                   // delta rule: a1 and g1 outputs, each padded with zeros to 64
    __shared__ __align__(16) float q[256], k[256], g[256];
    __shared__ float v[256], o[256], gate[256];
    const uint32_t h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane & 7, quads = l.pitch / 32;
    pdl_launch_dependents();
    // rows of the rank projections, eight lanes to a row (decays first, then the gate): weights, so their first kAhead words per
    // lane are fetched while the previous launch is still running
    constexpr uint32_t kAhead = kMaxQuads <= 4 ? 4 : 8;
    uint4 ahead[kAhead];
    const uint32_t words = kDelta ? (max(l.a2_ld, l.g2_ld) + 63) / 64 : 0;      // 16-byte words per lane and row
    auto rank_row = [&](uint32_t r, uint32_t& ld) -> const __nv_bfloat16* {     // null: padding
        const bool is_g = r >= l.pitch;
        const uint32_t d = is_g ? r - l.pitch : r;
        ld = is_g ? l.g2_ld : l.a2_ld;
        if (d >= (is_g ? l.vdim : l.dim)) return nullptr;
        return is_g ? l.g2 + static_cast<size_t>(h * l.vdim + d) * ld : l.a2 + static_cast<size_t>(h * l.dim + d) * ld;
    };
    if (kDelta) {
        uint32_t r = warp * 4 + (lane >> 3), word = 0;
#pragma unroll
        for (uint32_t i = 0; i < kAhead; ++i) {
            uint32_t ld;
            const __nv_bfloat16* w = rank_row(r, ld);
            const uint32_t c = (word * 8 + part) * 8;
            ahead[i] = w && c < ld ? __ldg(reinterpret_cast<const uint4*>(w + c)) : make_uint4(0, 0, 0, 0);
            if (++word == words) { word = 0; r += kWarps * 4; }
        }
    }
    pdl_wait();
    // the first columns' state words are on their way while the token's vectors are formed
    float* const state = l.state + static_cast<size_t>(h) * l.vdim * l.pitch + part * 4;
    uint32_t col = warp * 4 + (lane >> 3);
    float4 pre[kMaxQuads];
#pragma unroll
    for (uint32_t i = 0; i < kMaxQuads; ++i)
        pre[i] = (i < quads && col < l.vdim) ? __ldcg(reinterpret_cast<const float4*>(state + static_cast<size_t>(col) * l.pitch + i * 32)) : make_float4(0.f, 0.f, 0.f, 0.f);
    float beta = 0.0f;
    if (kDelta) {
        const int pos = *pos_ptr;
        const uint32_t channels = linear_channels(l), kd = l.kv_heads * l.dim, qh = h / (l.heads / l.kv_heads);
        const uint32_t pad_a = (l.rank_a + 63) & ~63u;
        for (uint32_t i = threadIdx.x; i < step_low_floats(l); i += kStepThreads) {
            const bool is_g = i >= pad_a;
            const uint32_t c = is_g ? i - pad_a : i;
            low[i] = c < (is_g ? l.rank_g : l.rank_a) ? __ldcg(proj + channels + l.heads + (is_g ? l.rank_a : 0u) + c) : 0.0f;
        }
        beta = logistic(__ldcg(proj + channels + h));
        const bool owner = h % (l.heads / l.kv_heads) == 0;        // one CTA per q/k head keeps its ring
        float* slot = l.ring + static_cast<size_t>(static_cast<uint32_t>(pos) % l.taps) * channels;
        for (uint32_t i = threadIdx.x; i < 2 * l.pitch + l.vdim; i += kStepThreads) {
            const bool is_v = i >= 2 * l.pitch, is_k = !is_v && i >= l.pitch;
            const uint32_t d = is_v ? i - 2 * l.pitch : is_k ? i - l.pitch : i;
            float y = 0.0f;
            if (is_v || d < l.dim) {
                const uint32_t c = is_v ? 2 * kd + h * l.vdim + d : (is_k ? kd : 0u) + qh * l.dim + d;
                y = conv_silu(l, proj, 0, 0, pos, c, channels);
                if (is_v || owner) slot[c] = __ldcg(proj + c);
            }
            (is_v ? v : is_k ? k : q)[d] = y;
        }
        __syncthreads();
        // decays and output gate
        const float a_scale = -expf(l.a_log[h]);
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
            if (part == 0 && r < l.pitch + l.vdim) {
                if (is_g) gate[r - l.pitch] = logistic(acc);
                else g[r] = r < l.dim ? expf(a_scale * softplus_f(acc + l.dt_bias[h * l.dim + r])) : 0.0f;
            }
            acc = 0.0f;
            word = 0;
            r += kWarps * 4;
        };
        // r - lane / 8 and word are the same in all lanes of a warp, so the loops below do not diverge around the shuffles
#pragma unroll
        for (uint32_t i = 0; i < kAhead; ++i)
            if (r - (lane >> 3) < l.pitch + l.vdim) take(ahead[i]);
        while (r - (lane >> 3) < l.pitch + l.vdim) {
            uint32_t ld;
            const __nv_bfloat16* w = rank_row(r, ld);
            const uint32_t c = (word * 8 + part) * 8;
            take(w && c < ld ? __ldg(reinterpret_cast<const uint4*>(w + c)) : make_uint4(0, 0, 0, 0));
        }
        __syncthreads();
        if (warp < 2) {                                            // unit norms: warp 0 takes q, warp 1 k
            float* x = warp ? k : q;
            float ss = 0.0f;
            for (uint32_t d = lane; d < l.pitch; d += 32) ss += x[d] * x[d];
            float inv = 1.0f / sqrtf(warp_sum(ss) + kUnitEps);
            if (!warp) inv *= 1.0f / sqrtf(static_cast<float>(l.dim));
            for (uint32_t d = lane; d < l.pitch; d += 32) x[d] *= inv;
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
    for (uint32_t i = threadIdx.x; i < l.vdim; i += kStepThreads) out[h * l.vdim + i] = o[i] * inv * l.norm[i] * (kDelta ? gate[i] : 1.0f);
}

}  // namespace zk
