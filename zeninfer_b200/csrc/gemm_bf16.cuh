// Products of bfloat16 matrices with a block of tokens.
//
// gemm_bf16_kernel: tcgen05.mma kind::f16, bf16 x bf16 -> fp32.  Weight rows are M (128 per tile), tokens are N (kNTile), so that
// a TMEM lane is a weight row and consecutive lanes store consecutive outputs of one token.  One persistent CTA per SM, six warps:
// TMA producer (64 columns of K per stage: 128 x 128 B of weights and kNTile x 128 B of activations, 128-byte swizzle), MMA issuer,
// four epilogue warps; two accumulators in TMEM, so the epilogue of a tile runs under the next tile's products.  K and rows that
// do not fill a tile arrive as zeros from the tensor maps.  The first 2 pairs rows may be (gate, up) pairs that leave as
// silu(gate) * up: neighbouring TMEM lanes, exchanged between lanes of the epilogue warp.
//
// gemm_bf16_exact_kernel: fp32 activations times bf16 weights in fp32 FMAs, for the 32-bit mode.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include "gemv_bf16.cuh"

namespace zk {

constexpr int kBgM = 128, kBgK = 64;                       // tile rows; K columns per stage (128 bytes)
constexpr int kBgThreads = 6 * 32;
constexpr uint32_t kBgABytes = kBgM * kBgK * 2;

struct GemmBf16Params {
    CUtensorMap map_w;        // [rows][ld] bf16, box 64 x 128
    CUtensorMap map_x;        // [tokens][ld] bf16, box 64 x kNTile
    float* out;               // [tokens][out_ld] fp32, or null; row r of the matrix is column r - 2 pairs
    __nv_bfloat16* out_bf16;  // [tokens][out_ld] bf16 when out is null
    __nv_bfloat16* gated;     // [tokens][gated_ld]: column i from rows 2 i and 2 i + 1
    const float* bias;        // [rows - 2 pairs], or null
    uint32_t out_ld, gated_ld, pairs, rows, tokens, k_tiles, m_tiles, n_tiles;
    int act;
    float cap;
    int* error_word;
};

template <int kNTile>
__host__ __device__ constexpr int gemm_bf16_stages() { return kNTile == 256 ? 4 : kNTile == 128 ? 6 : 8; }
template <int kNTile>
__host__ __device__ constexpr uint32_t gemm_bf16_stage_bytes() { return kBgABytes + kNTile * kBgK * 2; }
template <int kNTile>
__host__ __device__ constexpr uint32_t gemm_bf16_smem_bytes() { return 1024 + gemm_bf16_stages<kNTile>() * gemm_bf16_stage_bytes<kNTile>() + 256; }

// Instruction descriptor, kind::f16: bf16 x bf16 -> fp32, both operands K-major, dense.
__host__ __device__ constexpr uint32_t umma_idesc_bf16(uint32_t m, uint32_t n) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((n >> 3) << 17) | ((m >> 4) << 24);
}
__device__ __forceinline__ void tc_mma_f16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{ .reg .pred p; setp.ne.b32 p, %4, 0; tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }"
        ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}

template <int kNTile>
__global__ void __launch_bounds__(kBgThreads, 1) gemm_bf16_kernel(const __grid_constant__ GemmBf16Params p) {
    constexpr int kStages = gemm_bf16_stages<kNTile>();
    constexpr uint32_t kStageBytes = gemm_bf16_stage_bytes<kNTile>();
    constexpr uint32_t kTmemCols = 2 * kNTile < 32 ? 32 : 2 * kNTile;
    extern __shared__ uint8_t bg_smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(bg_smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + kStages * kStageBytes);
    uint64_t* empty = full + kStages;
    uint64_t* tmem_full = empty + kStages;
    uint64_t* tmem_empty = tmem_full + 2;
    uint32_t* tmem_base_slot = reinterpret_cast<uint32_t*>(tmem_empty + 2);
    volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_base_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&tmem_full[b], 1); mbar_init(&tmem_empty[b], 4); }
        *abort_word = 0;
        mbar_fence_init();
        tma_prefetch_descriptor(&p.map_w);
        tma_prefetch_descriptor(&p.map_x);
    }
    if (warp == 1) tmem_alloc(tmem_base_slot, kTmemCols);
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_base_slot, tiles = p.m_tiles * p.n_tiles;
    pdl_launch_dependents();

    if (warp == 0) {
        if (lane == 0) {
            pdl_wait();                                    // the activations are the previous launch's
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x) {
                const int m0 = static_cast<int>((tile / p.n_tiles) * kBgM), n0 = static_cast<int>((tile % p.n_tiles) * kNTile);
                for (uint32_t kt = 0; kt < p.k_tiles; ++kt, ++it) {
                    const uint32_t stage = it % kStages;
                    if (it >= kStages && !mbar_wait(&empty[stage], ((it / kStages) - 1) & 1)) {
                        *abort_word = 1; atomicExch(p.error_word, kErrEmptyWaitTimeout); ok = false;
                    }
                    if (*abort_word) ok = false;
                    if (!ok) break;
                    uint8_t* st = smem + stage * kStageBytes;
                    mbar_arrive_expect_tx(&full[stage], kStageBytes);
                    tma_load_2d(st, &p.map_w, static_cast<int>(kt * kBgK), m0, &full[stage]);
                    tma_load_2d(st + kBgABytes, &p.map_x, static_cast<int>(kt * kBgK), n0, &full[stage]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(kBgM, kNTile);
            uint32_t it = 0, count = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x, ++count) {
                const uint32_t set = count & 1;
                if (count >= 2) {
                    if (!mbar_wait(&tmem_empty[set], ((count >> 1) - 1) & 1)) {
                        *abort_word = 1; atomicExch(p.error_word, kErrTmemWaitTimeout);
                        break;
                    }
                    tc_fence_after_sync();
                }
                for (uint32_t kt = 0; kt < p.k_tiles; ++kt, ++it) {
                    const uint32_t stage = it % kStages;
                    if (*abort_word || !mbar_wait(&full[stage], (it / kStages) & 1)) {
                        if (!*abort_word) { *abort_word = 1; atomicExch(p.error_word, kErrFullWaitTimeout); }
                        ok = false;
                        break;
                    }
                    tc_fence_after_sync();
                    const uint32_t base = smem_u32(smem + stage * kStageBytes);
                    const uint64_t a = umma_desc_k_sw128(base), b = umma_desc_k_sw128(base + kBgABytes);
#pragma unroll
                    for (uint32_t j = 0; j < 4; ++j)           // 16 columns = 32 bytes = two 16-byte units further into the swizzle atom
                        tc_mma_f16(tmem_base + set * kNTile, a + 2 * j, b + 2 * j, idesc, (kt | j) ? 1u : 0u);
                    tc_commit(&empty[stage]);
                }
                if (ok) tc_commit(&tmem_full[set]);
            }
        }
    } else {
        const uint32_t quad = static_cast<uint32_t>(warp) & 3;     // the TMEM lanes a warp may touch: 32 * (warp id % 4)
        uint32_t count = 0;
        pdl_wait();                                                // the outputs may still be read by an earlier launch
        for (uint32_t tile = blockIdx.x; tile < tiles; tile += gridDim.x, ++count) {
            const uint32_t set = count & 1, n0 = (tile % p.n_tiles) * kNTile, r = (tile / p.n_tiles) * kBgM + quad * 32 + lane, paired = 2 * p.pairs;
            const float bias = p.bias && r >= paired && r < p.rows ? __ldg(p.bias + r - paired) : 0.0f;
            if (*abort_word || !mbar_wait(&tmem_full[set], (count >> 1) & 1)) {
                if (lane == 0 && !*abort_word) { *abort_word = 1; atomicExch(p.error_word, kErrTmemWaitTimeout); }
                break;
            }
            tc_fence_after_sync();
            constexpr int kChunk = kNTile < 32 ? 16 : 32;
#pragma unroll 1
            for (uint32_t c0 = 0; c0 < static_cast<uint32_t>(kNTile); c0 += kChunk) {
                uint32_t v[kChunk];
                const uint32_t addr = tmem_base + set * kNTile + c0 + ((quad * 32) << 16);
                if constexpr (kChunk == 32) tmem_ld_32x32(addr, v); else tmem_ld_32x16(addr, v);
                tmem_ld_wait();
                if (c0 + kChunk == static_cast<uint32_t>(kNTile)) {
                    tc_fence_before_sync();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(&tmem_empty[set]);
                }
                if (r - lane < paired) {                           // some of the warp's rows are pairs: an even lane takes one token, its partner the next
                    const bool odd = lane & 1;
#pragma unroll
                    for (int c = 0; c < kChunk; c += 2) {
                        const float keep = __uint_as_float(odd ? v[c + 1] : v[c]);
                        const float other = __shfl_xor_sync(0xffffffffu, __uint_as_float(odd ? v[c] : v[c + 1]), 1);
                        const uint32_t t = n0 + c0 + c + (odd ? 1u : 0u);
                        if (r < paired && t < p.tokens) p.gated[static_cast<size_t>(t) * p.gated_ld + r / 2] = __float2bfloat16_rn(odd ? silu_f(other) * keep : silu_f(keep) * other);
                    }
                }
                if (r >= paired && r < p.rows) {
#pragma unroll
                    for (int c = 0; c < kChunk; ++c) {
                        const uint32_t t = n0 + c0 + c;
                        if (t < p.tokens) {
                            const float y = dense_activation(__uint_as_float(v[c]) + bias, p.act, p.cap);
                            const size_t at = static_cast<size_t>(t) * p.out_ld + (r - paired);
                            if (p.out) p.out[at] = y; else p.out_bf16[at] = __float2bfloat16_rn(y);
                        }
                    }
                }
            }
        }
    }
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem_base, kTmemCols);
    }
}

// out[t][r - 2 pairs] = act(sum_k x[t][k] w[r][k] + bias[r - 2 pairs]) and gated[t][i] = silu(row 2 i) * (row 2 i + 1), 64 x 64 sums per
// CTA, four by four per thread.
constexpr int kExactTile = 64, kExactK = 16;
__global__ void __launch_bounds__(256) gemm_bf16_exact_kernel(const __nv_bfloat16* __restrict__ w, uint32_t w_ld, const float* __restrict__ x, uint32_t x_ld,
                                                              float* __restrict__ out, uint32_t out_ld, uint32_t rows, uint32_t tokens, uint32_t K, int act,
                                                              float cap, const float* __restrict__ bias, float* __restrict__ gated, uint32_t gated_ld, uint32_t pairs) {
    __shared__ float ws[kExactK][kExactTile + 4], xs[kExactK][kExactTile + 4];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t r0 = blockIdx.x * kExactTile, t0 = blockIdx.y * kExactTile, tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < K; k0 += kExactK) {
        for (uint32_t i = threadIdx.x; i < kExactTile * kExactK; i += 256) {
            const uint32_t row = i / kExactK, k = i % kExactK;
            ws[k][row] = (r0 + row < rows && k0 + k < K) ? __bfloat162float(w[static_cast<size_t>(r0 + row) * w_ld + k0 + k]) : 0.0f;
            xs[k][row] = (t0 + row < tokens && k0 + k < K) ? x[static_cast<size_t>(t0 + row) * x_ld + k0 + k] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kExactK; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = ws[k][tx * 4 + i]; b[i] = xs[k][ty * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const uint32_t t = t0 + ty * 4 + j;
        if (t >= tokens) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t r = r0 + tx * 4 + i;
            if (r < 2 * pairs) {
                if (!(i & 1)) gated[static_cast<size_t>(t) * gated_ld + r / 2] = silu_f(acc[i][j]) * acc[i + 1 < 4 ? i + 1 : i][j];
            } else if (r < rows) {
                out[static_cast<size_t>(t) * out_ld + (r - 2 * pairs)] = dense_activation(acc[i][j] + (bias ? __ldg(bias + r - 2 * pairs) : 0.0f), act, cap);
            }
        }
    }
}

}  // namespace zk
