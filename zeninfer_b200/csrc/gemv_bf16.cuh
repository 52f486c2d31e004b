// Decode-time products of bfloat16 matrices with one fp32 vector, memory-bound by design.
//
//   * one CTA per SM owns a contiguous slice of the launch's rows (over all its tensors); its sixteen warps split K in units of
//     256 columns (and, where K has fewer units than warps, the row groups too), eight rows per step: a lane holds 16 bytes of
//     each of eight rows and eight values of x, and two steps' loads (sixteen 16-byte words per lane) are in flight;
//   * weights are constants: the first two steps' loads go out before the previous grid has finished (griddepcontrol);
//   * the prologue can finish the sublayer before it (row_ops.cuh: grouped norm, residual add, token shift or output norm), so
//     a decode step needs no launches for them: every CTA forms the input vector itself, CTA 0 stores the residual stream;
//   * the epilogue adds a bias and applies the product's activation (squared ReLU, or the logits' soft cap) in fp32; a matrix may
//     begin with pairs of rows (gate, up) that leave the launch as silu(gate) * up.
// Activations are fp32 throughout: the product is exact up to fp32 accumulation.
#pragma once
#include "row_ops.cuh"

namespace zk {

constexpr int kDenseThreads = 512, kDenseWarps = kDenseThreads / 32;
constexpr uint32_t kDenseUnit = 256;          // columns a warp takes at a time: eight per lane
constexpr int kDenseRows = 8;                 // rows per step
constexpr int kDenseMaxTasks = 4;

enum : int { kActNone = 0, kActSquaredRelu = 1, kActSoftcap = 2 };

struct DenseTask {
    const __nv_bfloat16* w;   // [rows][ld], zero beyond the real columns
    const float* x;           // [K]; ignored when the launch carries a prologue
    float* y;                 // [rows - 2 pairs]
    const float* bias;        // [rows - 2 pairs], or null
    float* gated;             // [pairs]
    uint32_t rows, K, ld;
    uint32_t first_row;       // index of its first row in the launch's row space
    uint32_t pairs;           // rows 2 i and 2 i + 1 (i < pairs) give gated[i]; first_row is even then
    int act;
    float cap;
};

struct DenseGemvParams {
    DenseTask task[kDenseMaxTasks];
    uint32_t tasks, total_rows;
    uint32_t k_split;         // warps that share a row group: a power of two, at most kDenseWarps
    uint32_t row_unit;        // a CTA's slice begins at a multiple of this many rows: 2 where a task has pairs
    uint32_t has_prologue;    // 1: one task, whose input is the prologue's view
    uint32_t scratch_floats;
    SublayerEnd pre;
};

__host__ __device__ inline uint32_t dense_units(uint32_t ld) { return (ld + kDenseUnit - 1) / kDenseUnit; }

__device__ __forceinline__ float dense_activation(float v, int act, float cap) {
    if (act == kActSquaredRelu) { const float r = fmaxf(v, 0.0f); return r * r; }
    if (act == kActSoftcap) return cap * tanhf(v / cap);
    return v;
}
__device__ __forceinline__ void dense_fma8(const uint4& w, const float (&x)[8], float& acc) {
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        acc = fmaf(__uint_as_float(u[i] << 16), x[2 * i], acc);
        acc = fmaf(__uint_as_float(u[i] & 0xffff0000u), x[2 * i + 1], acc);
    }
}

__global__ void __launch_bounds__(kDenseThreads, 1) gemv_bf16_kernel(const __grid_constant__ DenseGemvParams p) {
    extern __shared__ __align__(16) float dense_smem[];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint64_t row_units = (p.total_rows + p.row_unit - 1) / p.row_unit;
    const uint32_t slice0 = static_cast<uint32_t>(row_units * blockIdx.x / gridDim.x) * p.row_unit;
    const uint32_t slice1 = min(static_cast<uint32_t>(row_units * (blockIdx.x + 1) / gridDim.x) * p.row_unit, p.total_rows);
    const uint32_t team = warp / p.k_split, part = warp % p.k_split, teams = kDenseWarps / p.k_split;
    pdl_launch_dependents();

    // a warp's steps: (task, row group, K unit), walked in that order
    struct Walk { uint32_t ti, r, r_end, u; };
    auto enter = [&](Walk& w) {      // the next task of the slice with work for this warp
        for (; w.ti < p.tasks; ++w.ti) {
            const DenseTask& t = p.task[w.ti];
            const uint32_t a = max(slice0, t.first_row), b = min(slice1, t.first_row + t.rows);
            if (a < b && a + team * kDenseRows < b && part < dense_units(t.ld)) {
                w.r = a - t.first_row + team * kDenseRows;
                w.r_end = b - t.first_row;
                w.u = part;
                return;
            }
        }
    };
    auto load = [&](const Walk& w, uint4 (&v)[kDenseRows]) {
        const DenseTask& t = p.task[w.ti];
        const uint32_t col = w.u * kDenseUnit + lane * 8;
        const __nv_bfloat16* base = t.w + static_cast<size_t>(w.r) * t.ld + col;
#pragma unroll
        for (int i = 0; i < kDenseRows; ++i)
            v[i] = (w.r + i < w.r_end && col < t.ld) ? __ldg(reinterpret_cast<const uint4*>(base + static_cast<size_t>(i) * t.ld)) : make_uint4(0, 0, 0, 0);
    };
    auto advance = [&](Walk& w) {    // to the step after w
        const bool row_done = w.u + p.k_split >= dense_units(p.task[w.ti].ld);
        w.u += p.k_split;
        if (row_done) {
            w.u = part;
            w.r += teams * kDenseRows;
            if (w.r >= w.r_end) { ++w.ti; enter(w); }
        }
    };
    // two steps' weights are in flight at any time: while one buffer is used up, the other's loads are on their way
    uint4 buf0[kDenseRows], buf1[kDenseRows];
    Walk w0{0, 0, 0, 0}, w1;
    enter(w0);
    if (w0.ti < p.tasks) load(w0, buf0);
    w1 = w0;
    if (w1.ti < p.tasks) advance(w1);
    if (w1.ti < p.tasks) load(w1, buf1);

    // the input vectors in shared memory, each padded with zeros to whole units; then per-row partial sums of the slice
    float* xs = dense_smem;
    uint32_t x_floats = 0;
    pdl_wait();
    if (p.has_prologue) {
        x_floats = dense_units(p.task[0].ld) * kDenseUnit;
        float* scratch = dense_smem + x_floats;
        sublayer_row<kDenseThreads>(p.pre, 0, xs, scratch);
        if (blockIdx.x == 0) {
            if (p.pre.x_out)
                for (uint32_t i = threadIdx.x; i < p.pre.n; i += kDenseThreads) p.pre.x_out[i] = xs[i];
            if (p.pre.keep)
                for (uint32_t i = threadIdx.x; i < p.pre.n; i += kDenseThreads) p.pre.keep[i] = p.pre.x_in[i];
        }
        for (uint32_t i = p.pre.n + threadIdx.x; i < x_floats; i += kDenseThreads) xs[i] = 0.0f;
        sublayer_view<kDenseThreads>(p.pre, xs, p.pre.before, scratch);
    } else {
        for (uint32_t ti = 0; ti < p.tasks; ++ti) {
            const DenseTask& t = p.task[ti];
            const uint32_t padded = dense_units(t.ld) * kDenseUnit;
#pragma unroll 8
            for (uint32_t i = threadIdx.x; i < padded; i += kDenseThreads) xs[x_floats + i] = i < t.K ? __ldcg(t.x + i) : 0.0f;
            x_floats += padded;
        }
        __syncthreads();
    }
    float* sums = dense_smem + x_floats + p.scratch_floats;      // [rows of the slice][k_split]

    float acc[kDenseRows];
#pragma unroll
    for (int i = 0; i < kDenseRows; ++i) acc[i] = 0.0f;
    auto consume = [&](const Walk& at, const uint4 (&w)[kDenseRows]) {
        const DenseTask& t = p.task[at.ti];
        uint32_t x_base = 0;                                      // where the task's input starts in xs
        for (uint32_t i = 0; i < at.ti; ++i) x_base += dense_units(p.task[i].ld) * kDenseUnit;
        const float4* xv = reinterpret_cast<const float4*>(xs + x_base + at.u * kDenseUnit + lane * 8);
        const float4 x0 = xv[0], x1 = xv[1];
        const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
        for (int i = 0; i < kDenseRows; ++i) dense_fma8(w[i], x, acc[i]);
        if (at.u + p.k_split < dense_units(t.ld)) return;
        // the row group is done: eight sums over 32 lanes; at each of the first three exchanges a lane keeps half of the rows it carries
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const bool hi = lane & 16;
            const float keep = hi ? acc[i + 4] : acc[i], give = hi ? acc[i] : acc[i + 4];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, 16);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const bool hi = lane & 8;
            const float keep = hi ? acc[i + 2] : acc[i], give = hi ? acc[i] : acc[i + 2];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, 8);
        }
        {
            const bool hi = lane & 4;
            const float keep = hi ? acc[1] : acc[0], give = hi ? acc[0] : acc[1];
            acc[0] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
        }
        acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 2);
        acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
        const uint32_t mine = ((lane >> 4) & 1) * 4 + ((lane >> 3) & 1) * 2 + ((lane >> 2) & 1);
        if ((lane & 3) == 0 && at.r + mine < at.r_end) sums[static_cast<size_t>(t.first_row + at.r + mine - slice0) * p.k_split + part] = acc[0];
#pragma unroll
        for (int i = 0; i < kDenseRows; ++i) acc[i] = 0.0f;
    };
    while (w0.ti < p.tasks) {
        consume(w0, buf0);
        w0 = w1;
        if (w0.ti < p.tasks) advance(w0);
        if (w0.ti < p.tasks) load(w0, buf0);
        if (w1.ti >= p.tasks) break;
        consume(w1, buf1);
        w1 = w0;
        if (w1.ti < p.tasks) advance(w1);
        if (w1.ti < p.tasks) load(w1, buf1);
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < slice1 - slice0; i += kDenseThreads) {
        const uint32_t row = slice0 + i;
        uint32_t ti = 0;
        while (row >= p.task[ti].first_row + p.task[ti].rows) ++ti;
        const DenseTask& t = p.task[ti];
        const uint32_t parts = min(p.k_split, dense_units(t.ld));
        auto total = [&](uint32_t at) {
            float v = 0.0f;
            for (uint32_t s = 0; s < parts; ++s) v += sums[static_cast<size_t>(at) * p.k_split + s];
            return v;
        };
        const uint32_t r = row - t.first_row, paired = 2 * t.pairs;
        if (r < paired) {
            if (!(r & 1)) t.gated[r / 2] = silu_f(total(i)) * total(i + 1);
        } else {
            t.y[r - paired] = dense_activation(total(i) + (t.bias ? __ldg(t.bias + r - paired) : 0.0f), t.act, t.cap);
        }
    }
}

}  // namespace zk
