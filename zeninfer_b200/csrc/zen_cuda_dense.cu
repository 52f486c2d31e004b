// C-ABI of the bfloat16 decoders' kernels (include/zen_cuda.h): argument checks, tensor maps and launches.
#include "../../include/zen_cuda.h"

#include <cuda.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <string>
#include <type_traits>

#include "attention.cuh"
#include "gemm_bf16.cuh"
#include "gemv_bf16.cuh"
#include "host_state.h"
#include "linear_state.cuh"
#include "row_ops.cuh"

namespace zk_host {
bool set_dense_wait_budget(long long cycles) { return cudaMemcpyToSymbol(zk::g_wait_budget_cycles, &cycles, sizeof cycles) == cudaSuccess; }
}  // namespace zk_host

namespace {

using zk_host::Entry;

template <typename... KArgs, typename... Args>
cudaError_t launch(const Entry& e, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    if (smem > 48 * 1024) {
        const cudaError_t r = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
        if (r != cudaSuccess) return r;
    }
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = e.stream;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = e.pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

bool is_bf16(const zen_cuda_weights* w) { return w && w->format == ZEN_CUDA_BF16; }
const __nv_bfloat16* plane(const zen_cuda_weights* w) { return static_cast<const __nv_bfloat16*>(w->plane[0]); }
uint32_t u32(size_t v) { return static_cast<uint32_t>(v); }
uint32_t pitch32(uint32_t n) { return (n + 31u) & ~31u; }

bool sublayer_ok(const zen_cuda_sublayer_end* s) {
    if (!s || !s->x_in || !s->n || !s->groups || s->n % s->groups || s->groups > 4096) return false;
    if (s->x_out == s->x_in || (s->y_b && (!s->y_a || !s->norm_weight || !s->weight_a || !s->weight_b))) return false;
    return !(s->shift && (!s->before || s->out_norm || s->before == s->keep));
}
zk::SublayerEnd device_form(const zen_cuda_sublayer_end& s) {
    return zk::SublayerEnd{s.x_in, s.x_out, s.y_a, s.y_b, s.weight_a, s.weight_b, s.norm_weight, s.keep, s.shift, s.before, s.out_norm, s.n, s.groups, s.eps};
}

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                   const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// [outer][pitch] bf16, boxes of 64 columns x box_rows, 128-byte swizzle; what lies outside reads as zero.
bool map_bf16(const Entry& e, CUtensorMap* map, const void* base, uint64_t inner, uint64_t outer, uint64_t pitch, uint32_t box_rows) {
    const cuuint64_t dims[2] = {inner, outer};
    const cuuint64_t strides[1] = {pitch * 2};
    const cuuint32_t box[2] = {zk::kBgK, box_rows}, step[2] = {1, 1};
    return reinterpret_cast<EncodeTiledFn>(e.encode_tiled)(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, step,
                                                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int kNTile>
cudaError_t launch_gemm(const Entry& e, zk::GemmBf16Params& p) {
    const uint32_t tiles = p.m_tiles * p.n_tiles;
    return launch(e, zk::gemm_bf16_kernel<kNTile>, dim3(std::min<uint32_t>(tiles, u32(e.sm_count))), dim3(zk::kBgThreads), zk::gemm_bf16_smem_bytes<kNTile>(), p);
}

bool window_ok(const zen_cuda_window_attention* a) {
    return a && a->heads && a->kv_heads && a->heads % a->kv_heads == 0 && a->qk_dim && a->v_dim && a->pitch == pitch32(std::max(a->qk_dim, a->v_dim)) &&
           a->pitch <= 256 && a->window && a->max_positions && a->k_cache && a->v_cache && !a->q_weight == !a->k_weight &&
           (a->q_weight ? !a->taps && !a->rot_pairs && !a->v_first && !a->v_keep
                        : 2 * a->rot_pairs <= a->qk_dim && (!a->rot_pairs || (a->rot_cos && a->rot_sin)) && (!a->taps || (a->conv && a->ring)));
}
bool is_rotary(const zen_cuda_window_attention& a) { return !a.q_weight; }
zk::AttnWindow device_form(const zen_cuda_window_attention& a, const float* gate) {
    zk::AttnWindow w{a.keep_first, a.bias ? 1u : 0u, a.q_weight, a.k_weight, gate, a.eps, a.qk_dim, a.v_dim, a.gate_values ? 1u : 0u, {}};
    w.rotary.conv = zk::ShortConv{a.conv, a.ring, a.taps, (a.heads + a.kv_heads) * a.qk_dim + a.kv_heads * a.v_dim};
    w.rotary.turn = zk::HalfRotation{a.rot_cos, a.rot_sin, a.rot_pairs, a.max_positions};
    w.rotary.v_first = a.v_first;
    w.rotary.v_keep = a.v_keep;
    w.rotary.share = a.v_share;
    return w;
}

bool linear_ok(const zen_cuda_linear_layer* l, int rule) {
    if (!l || rule < ZEN_CUDA_STATE_GATED_WRITE || rule > ZEN_CUDA_STATE_DECAYED_WRITE || !l->heads || !l->dim || !l->vdim || l->dim > 256 || l->vdim > 256 || !l->state || !l->norm) return false;
    if (rule == ZEN_CUDA_STATE_GATED_WRITE) return l->kv_heads == l->heads && l->f_bias && l->lower;
    if (rule == ZEN_CUDA_STATE_DECAYED_WRITE)
        return l->kv_heads == l->heads && 2 * l->rot_pairs <= l->dim && (!l->rot_pairs || (l->rot_cos && l->rot_sin && l->max_positions)) &&
               (l->decay || (l->dt_bias && l->inv_tau > 0.0f && is_bf16(l->a2) && l->a2->rows == size_t(l->heads) * l->dim && l->a2->cols <= 512));
    return l->kv_heads && l->heads % l->kv_heads == 0 && l->taps && l->conv && l->a_log && l->dt_bias && l->ring && is_bf16(l->a2) && is_bf16(l->g2) &&
           l->a2->rows == size_t(l->heads) * l->dim && l->g2->rows == size_t(l->heads) * l->vdim;
}
zk::LinearLayer device_form(const zen_cuda_linear_layer& l, int rule) {
    zk::LinearLayer d{};
    d.heads = l.heads; d.kv_heads = l.kv_heads; d.dim = l.dim; d.vdim = l.vdim; d.pitch = pitch32(l.dim);
    d.eps = l.eps; d.norm = l.norm; d.state = l.state;
    if (rule == ZEN_CUDA_STATE_DELTA_RULE) {
        d.conv = zk::ShortConv{l.conv, l.ring, l.taps, zk::linear_channels(d)};
        d.rank_a = u32(l.a2->cols); d.rank_g = u32(l.g2->cols); d.a2_ld = l.a2->nbp; d.g2_ld = l.g2->nbp;
        d.a_log = l.a_log; d.dt_bias = l.dt_bias; d.a2 = plane(l.a2); d.g2 = plane(l.g2);
    } else if (rule == ZEN_CUDA_STATE_DECAYED_WRITE) {
        d.turn = zk::HalfRotation{l.rot_cos, l.rot_sin, l.rot_pairs, l.max_positions};
        d.decay = l.decay;
        if (!l.decay) { d.rank_a = u32(l.a2->cols); d.a2_ld = l.a2->nbp; d.dt_bias = l.dt_bias; d.a2 = plane(l.a2); d.inv_tau = l.inv_tau; }
    } else {
        d.f_bias = l.f_bias; d.lower = l.lower;
    }
    return d;
}

// The groups' records, then the walk over them.
cudaError_t run_scan(Entry& e, int rule, uint32_t dim, const zk::ScanParams& p, const zk::LinearLayer& l) {
    const dim3 grid((p.vdim + zk::kScanColumns - 1) / zk::kScanColumns, p.heads);
    // A grid that fits the SMs one CTA each asks for more than half an SM's shared memory: launched while the groups kernel drains,
    // its CTAs would otherwise pile up on the first SMs to come free, and each runs for the whole block of tokens.
    const bool spread = static_cast<uint64_t>(grid.x) * grid.y <= static_cast<uint64_t>(e.sm_count);
    auto alone = [&](size_t smem) { return spread ? std::max(smem, e.smem_optin / 2 + 1024) : smem; };
    auto go = [&](auto quads, auto which) {
        constexpr int kQ = decltype(quads)::value, kRule = decltype(which)::value;
        constexpr bool kDelta = kRule == zk::kDeltaRule;
        const dim3 prepare(u32(((p.tokens + zk::kGroup - 1) / zk::kGroup * p.heads + 3) / 4));
        const size_t low = rule == ZEN_CUDA_STATE_DECAYED_WRITE ? size_t(4) * zk::kGroup * ((l.rank_a + 7) & ~7u) * sizeof(float) : 0;
        const cudaError_t first = launch(e, zk::state_groups_kernel<kQ, kRule>, prepare, dim3(128), low, p, l);
        if (!e.leave(first, "state_scan: groups")) return first;
        return launch(e, zk::state_scan_kernel<kQ, kDelta>, grid, dim3(zk::kScanThreads), alone(zk::scan_smem_bytes<kQ, kDelta>()), p);
    };
    auto by_rule = [&](auto quads) {
        return rule == ZEN_CUDA_STATE_DELTA_RULE      ? go(quads, std::integral_constant<int, zk::kDeltaRule>{})
               : rule == ZEN_CUDA_STATE_DECAYED_WRITE ? go(quads, std::integral_constant<int, zk::kDecayedWrite>{})
                                                      : go(quads, std::integral_constant<int, zk::kGatedWrite>{});
    };
    switch (pitch32(dim) / 32) {
    case 1: return by_rule(std::integral_constant<int, 1>{});
    case 2: return by_rule(std::integral_constant<int, 2>{});
    case 3: return by_rule(std::integral_constant<int, 3>{});
    case 4: return by_rule(std::integral_constant<int, 4>{});
    case 5: return by_rule(std::integral_constant<int, 5>{});
    case 6: return by_rule(std::integral_constant<int, 6>{});
    case 7: return by_rule(std::integral_constant<int, 7>{});
    default: return by_rule(std::integral_constant<int, 8>{});
    }
}

}  // namespace

#define ZC_ENTER(stream_arg, good, name)            \
    Entry e(stream_arg);                            \
    if (!e.ok) return 0;                            \
    if (!(good)) return e.fail(name ": bad arguments")

extern "C" {

int zen_cuda_dev_sublayer_end_rows(const zen_cuda_sublayer_end* end, size_t rows, void* d_view, size_t view_ld, int view_bf16, void* stream) {
    ZC_ENTER(stream, sublayer_ok(end) && rows && rows <= 65535 && (!d_view || view_ld >= end->n) && (d_view || end->x_out), "sublayer_end_rows");
    const zk::SublayerEnd p = device_form(*end);
    const size_t smem = (static_cast<size_t>(p.n) * (p.shift ? 2 : 1) + zk::row_scratch_floats(zk::kRowThreads, p.groups)) * sizeof(float);
    if (smem > e.smem_optin) return e.fail("sublayer_end_rows: the row does not fit shared memory");
    const cudaError_t r = view_bf16 ? launch(e, zk::sublayer_end_rows_kernel<__nv_bfloat16>, dim3(u32(rows)), dim3(zk::kRowThreads), smem, p,
                                             static_cast<__nv_bfloat16*>(d_view), u32(view_ld))
                                    : launch(e, zk::sublayer_end_rows_kernel<float>, dim3(u32(rows)), dim3(zk::kRowThreads), smem, p,
                                             static_cast<float*>(d_view), u32(view_ld));
    return e.leave(r, "sublayer_end_rows");
}

int zen_cuda_dev_dense_gemv(const zen_cuda_dense_task* tasks, size_t count, const zen_cuda_sublayer_end* pre, void* stream) {
    ZC_ENTER(stream, tasks && count && count <= zk::kDenseMaxTasks && (!pre || (count == 1 && sublayer_ok(pre))), "dense_gemv");
    static_assert(ZEN_CUDA_DENSE_MAX_TASKS == zk::kDenseMaxTasks, "task limit");
    zk::DenseGemvParams p{};
    uint64_t rows = 0;
    size_t x_floats = 0;
    uint32_t units = 1;
    p.row_unit = 1;
    for (size_t i = 0; i < count; ++i) {
        const zen_cuda_dense_task& t = tasks[i];
        if (!is_bf16(t.w) || (!pre && !t.d_x) || (pre && t.w->cols != pre->n) || (t.act == ZEN_CUDA_DENSE_SOFTCAP && !(t.cap > 0.0f)) ||
            t.gated_pairs > t.w->rows / 2 || (t.gated_pairs && (!t.d_gated || rows % 2)) || (t.w->rows > 2 * t.gated_pairs && !t.d_y))
            return e.fail("dense_gemv: bad task");
        p.task[i] = zk::DenseTask{plane(t.w), t.d_x, t.d_y, t.d_bias, t.d_gated, u32(t.w->rows), u32(t.w->cols), t.w->nbp, u32(rows), u32(t.gated_pairs), t.act, t.cap};
        if (t.gated_pairs) p.row_unit = 2;
        rows += t.w->rows;
        units = std::max(units, zk::dense_units(t.w->nbp));
        x_floats += static_cast<size_t>(zk::dense_units(t.w->nbp)) * zk::kDenseUnit;
    }
    if (rows > 0x7fffffffu) return e.fail("dense_gemv: too many rows");
    p.tasks = u32(count);
    p.total_rows = u32(rows);
    p.k_split = 1;
    while (p.k_split < static_cast<uint32_t>(zk::kDenseWarps) && p.k_split < units) p.k_split *= 2;
    if (pre) {
        p.has_prologue = 1;
        p.pre = device_form(*pre);
        p.scratch_floats = (zk::row_scratch_floats(zk::kDenseThreads, pre->groups) + 3u) & ~3u;
    }
    const uint32_t row_units = u32((rows + p.row_unit - 1) / p.row_unit), grid = std::min<uint32_t>(u32(e.sm_count), row_units);
    const size_t slice = static_cast<size_t>((row_units + grid - 1) / grid) * p.row_unit;
    const size_t smem = (x_floats + p.scratch_floats + slice * p.k_split) * sizeof(float);
    if (smem > e.smem_optin) return e.fail("dense_gemv: the input vector and a slice's sums do not fit shared memory");
    return e.leave(launch(e, zk::gemv_bf16_kernel, dim3(grid), dim3(zk::kDenseThreads), smem, p), "dense_gemv");
}

int zen_cuda_dev_dense_gemm(const zen_cuda_weights* w, const void* d_x, size_t x_ld, size_t tokens, void* d_out, size_t out_ld, int out_bf16,
                            const zen_cuda_dense_epilogue* epilogue, int exact, void* stream) {
    const zen_cuda_dense_epilogue ep = epilogue ? *epilogue : zen_cuda_dense_epilogue{};
    ZC_ENTER(stream, is_bf16(w) && d_x && tokens && tokens <= 0x7fffffffu && x_ld >= w->cols && ep.gated_pairs <= w->rows / 2 &&
                         (w->rows == 2 * ep.gated_pairs || (d_out && out_ld >= w->rows - 2 * ep.gated_pairs)) &&
                         (!ep.gated_pairs || (ep.d_gated && ep.gated_ld >= ep.gated_pairs)) && !(exact && out_bf16) &&
                         !(ep.act == ZEN_CUDA_DENSE_SOFTCAP && !(ep.cap > 0.0f)), "dense_gemm");
    if (exact) {
        const size_t ty = (tokens + zk::kExactTile - 1) / zk::kExactTile;
        if (ty > 65535) return e.fail("dense_gemm: too many tokens");
        return e.leave(launch(e, zk::gemm_bf16_exact_kernel, dim3(u32((w->rows + zk::kExactTile - 1) / zk::kExactTile), u32(ty)), dim3(256), 0, plane(w), w->nbp,
                              static_cast<const float*>(d_x), u32(x_ld), static_cast<float*>(d_out), u32(out_ld), u32(w->rows), u32(tokens), u32(w->cols), ep.act, ep.cap, ep.d_bias,
                              static_cast<float*>(ep.d_gated), u32(ep.gated_ld), u32(ep.gated_pairs)),
                       "dense_gemm");
    }
    if (x_ld % 8 || (reinterpret_cast<uintptr_t>(d_x) & 15)) return e.fail("dense_gemm: bf16 rows must be 16-byte aligned");
    if (!e.encode_tiled) return e.fail("dense_gemm: cuTensorMapEncodeTiled is not available");
    zk::GemmBf16Params p{};
    p.out = out_bf16 ? nullptr : static_cast<float*>(d_out);
    p.out_bf16 = out_bf16 ? static_cast<__nv_bfloat16*>(d_out) : nullptr;
    p.out_ld = u32(out_ld); p.rows = u32(w->rows); p.tokens = u32(tokens);
    p.k_tiles = u32((w->cols + zk::kBgK - 1) / zk::kBgK);
    p.m_tiles = u32((w->rows + zk::kBgM - 1) / zk::kBgM);
    p.act = ep.act; p.cap = ep.cap; p.bias = ep.d_bias; p.error_word = e.d_error;
    p.gated = static_cast<__nv_bfloat16*>(ep.d_gated); p.gated_ld = u32(ep.gated_ld); p.pairs = u32(ep.gated_pairs);
    // the tile width that moves the fewest operand bytes through the busiest SM
    int best = 0;
    uint64_t best_cost = ~0ull;
    for (int n : {256, 128, 64, 32}) {
        const uint64_t tiles = static_cast<uint64_t>(p.m_tiles) * ((tokens + n - 1) / n), waves = (tiles + e.sm_count - 1) / e.sm_count;
        const uint64_t cost = waves * static_cast<uint64_t>(zk::kBgM + n);
        if (cost < best_cost) { best_cost = cost; best = n; }
    }
    p.n_tiles = u32((tokens + best - 1) / best);
    // the matrix's padding columns are zeros, so the maps may end at the pitch; x is read up to its real columns only
    if (!map_bf16(e, &p.map_w, w->plane[0], w->nbp, w->rows, w->nbp, zk::kBgM) || !map_bf16(e, &p.map_x, d_x, w->cols, tokens, x_ld, u32(best)))
        return e.fail("dense_gemm: cuTensorMapEncodeTiled failed");
    const cudaError_t r = best == 256 ? launch_gemm<256>(e, p) : best == 128 ? launch_gemm<128>(e, p) : best == 64 ? launch_gemm<64>(e, p) : launch_gemm<32>(e, p);
    return e.leave(r, "dense_gemm");
}

int zen_cuda_dev_embed_rows_bf16(const zen_cuda_weights* embed, const zen_cuda_weights* positions, const int64_t* d_tokens, size_t tokens, const int* d_pos,
                                 float* d_out, void* stream) {
    ZC_ENTER(stream, is_bf16(embed) && (!positions || (is_bf16(positions) && positions->cols == embed->cols && d_pos)) && d_tokens && tokens && tokens <= 65535 && d_out,
             "embed_rows_bf16");
    return e.leave(launch(e, zk::embed_rows_bf16_kernel, dim3(u32((embed->cols + 255) / 256), u32(tokens)), dim3(256), 0, plane(embed), u32(embed->rows), embed->nbp,
                          positions ? plane(positions) : nullptr, positions ? u32(positions->rows) : 0u, positions ? positions->nbp : 0u,
                          reinterpret_cast<const long long*>(d_tokens), d_pos, d_out, u32(embed->cols), e.d_error),
                   "embed_rows_bf16");
}

int zen_cuda_dev_rows_view(const float* d_src, size_t src_ld, size_t n, size_t rows, void* d_dst, size_t ld, int bf16, void* stream) {
    ZC_ENTER(stream, d_src && d_dst && n && ld >= n && src_ld >= n && rows && rows <= 0x7fffffffu, "rows_view");
    const cudaError_t r = bf16 ? launch(e, zk::rows_view_kernel<__nv_bfloat16>, dim3(u32(rows)), dim3(256), 0, d_src, u32(src_ld), u32(n),
                                        static_cast<__nv_bfloat16*>(d_dst), u32(ld))
                               : launch(e, zk::rows_view_kernel<float>, dim3(u32(rows)), dim3(256), 0, d_src, u32(src_ld), u32(n), static_cast<float*>(d_dst), u32(ld));
    return e.leave(r, "rows_view");
}

int zen_cuda_dev_head_outputs_rows(const float* d_o, size_t rows, size_t heads, size_t width, size_t head_ld, const float* d_weight, float eps, const float* d_gate,
                                   size_t gate_ld, int gate_mode, void* d_dst, size_t ld, size_t fill, int bf16, void* stream) {
    ZC_ENTER(stream, d_o && rows && rows <= 0x7fffffffu && heads && width && head_ld >= width && gate_mode >= 0 && gate_mode <= 3 && (!gate_mode || d_gate) && d_dst &&
                         fill >= heads * width && ld >= fill, "head_outputs_rows");
    auto go = [&](auto* dst) {
        using T = std::remove_pointer_t<decltype(dst)>;
        return launch(e, zk::head_outputs_rows_kernel<T>, dim3(u32(rows)), dim3(256), 0, d_o, u32(heads), u32(width), u32(head_ld), d_weight, eps, d_gate, u32(gate_ld),
                      gate_mode, dst, u32(ld), u32(fill));
    };
    return e.leave(bf16 ? go(static_cast<__nv_bfloat16*>(d_dst)) : go(static_cast<float*>(d_dst)), "head_outputs_rows");
}

int zen_cuda_dev_window_attention_rows(const zen_cuda_window_attention* a, const float* d_proj_q, const float* d_proj_k, const float* d_proj_v, size_t ld,
                                       size_t tokens, const int* d_pos, float* d_q, float* d_out, void* stream) {
    ZC_ENTER(stream, window_ok(a) && d_proj_q && d_proj_k && d_proj_v && tokens && tokens <= 65535 && d_pos && d_q && d_out, "window_attention_rows");
    const zk::AttnWindow win = device_form(*a, nullptr);
    cudaError_t r;
    if (is_rotary(*a)) {
        const uint32_t items = a->heads + 2 * a->kv_heads, share = std::max(1u, std::min(64u, (items + 7) / 8));
        r = launch(e, zk::conv_rotary_append_rows_kernel, dim3(u32((tokens + zk::kStrip - 1) / zk::kStrip), share), dim3(256), 0, d_proj_q, d_proj_k, d_proj_v, u32(ld), win,
                   a->heads, a->kv_heads, a->pitch, u32(tokens), d_pos, d_q, a->k_cache, a->v_cache, a->max_positions, e.d_error);
        if (!e.leave(r, "window_attention_rows: append")) return 0;
        if (a->taps) {
            if (d_proj_k != d_proj_q + size_t(a->heads) * a->qk_dim || d_proj_v != d_proj_k + size_t(a->kv_heads) * a->qk_dim)
                return e.fail("window_attention_rows: the convolved q, k and v are consecutive columns");
            r = launch(e, zk::conv_ring_update_kernel, dim3((win.rotary.conv.channels + 255) / 256), dim3(256), 0, win.rotary.conv, d_proj_q, u32(ld), u32(tokens), d_pos);
            if (!e.leave(r, "window_attention_rows: ring")) return 0;
        }
    } else {
        r = launch(e, zk::qk_norm_append_rows_kernel, dim3(u32(tokens)), dim3(256), 0, d_proj_q, d_proj_k, d_proj_v, u32(ld), win, a->heads, a->kv_heads, a->pitch,
                   d_pos, d_q, a->k_cache, a->v_cache, a->max_positions, e.d_error);
        if (!e.leave(r, "window_attention_rows: append")) return 0;
    }
    const uint32_t group = a->heads / a->kv_heads;
    const int cap = a->pitch > 128 ? 2 : 4, r_heads = (cap >= 4 && group % 4 == 0) ? 4 : group % 2 == 0 ? 2 : 1;
    const size_t ctas = (tokens + zk::kPfTokens - 1) / zk::kPfTokens * a->kv_heads * (group / r_heads);
    if (ctas > 0x7fffffffu) return e.fail("window_attention_rows: too many tiles");
    auto go = [&](auto kernel) {
        return launch(e, kernel, dim3(u32(ctas)), dim3(zk::kPfThreads), 2 * 2 * zk::kPfBlock * a->pitch * sizeof(float), static_cast<const float*>(d_q),
                      static_cast<const float*>(a->k_cache), static_cast<const float*>(a->v_cache), d_pos, d_out, u32(tokens), a->heads, a->kv_heads, a->scale, a->window,
                      a->max_positions, e.d_error, win);
    };
    auto by_heads = [&](auto dim) {
        constexpr int kD = decltype(dim)::value;
        if constexpr (kD <= 128) {
            if (r_heads == 4) return go(zk::attention_prefill_kernel<kD, 4, true>);
        }
        return r_heads == 2 ? go(zk::attention_prefill_kernel<kD, 2, true>) : go(zk::attention_prefill_kernel<kD, 1, true>);
    };
    switch (a->pitch / 32) {
    case 1: r = by_heads(std::integral_constant<int, 32>{}); break;
    case 2: r = by_heads(std::integral_constant<int, 64>{}); break;
    case 3: r = by_heads(std::integral_constant<int, 96>{}); break;
    case 4: r = by_heads(std::integral_constant<int, 128>{}); break;
    case 5: r = by_heads(std::integral_constant<int, 160>{}); break;
    case 6: r = by_heads(std::integral_constant<int, 192>{}); break;
    case 7: r = by_heads(std::integral_constant<int, 224>{}); break;
    default: r = by_heads(std::integral_constant<int, 256>{}); break;
    }
    return e.leave(r, "window_attention_rows");
}

int zen_cuda_dev_window_attention_step(const zen_cuda_window_attention* a, const float* d_q, const float* d_k, const float* d_v, const float* d_gate, const int* d_pos,
                                       float* d_out, void* stream) {
    ZC_ENTER(stream, window_ok(a) && d_q && d_k && d_v && d_pos && d_out, "window_attention_step");
    auto go = [&](auto kernel) {
        return launch(e, kernel, dim3(zk::kAttnSplit, a->heads), dim3(zk::kAttnThreads), 0, d_q, static_cast<const float*>(nullptr), static_cast<const float*>(nullptr), d_pos,
                      d_out, a->heads, a->kv_heads, a->pitch, a->scale, a->window, a->max_positions, e.d_error, d_k, d_v, static_cast<const float*>(nullptr),
                      static_cast<const float*>(nullptr), 0u, a->k_cache, a->v_cache, device_form(*a, d_gate));
    };
    const bool wide = a->pitch > 128;
    const cudaError_t r = is_rotary(*a) ? (wide ? go(zk::attention_decode_kernel<true, true, zk::kAttnConvRotary>) : go(zk::attention_decode_kernel<true, false, zk::kAttnConvRotary>))
                                        : (wide ? go(zk::attention_decode_kernel<true, true, zk::kAttnNormed>) : go(zk::attention_decode_kernel<true, false, zk::kAttnNormed>));
    return e.leave(r, "window_attention_step");
}

int zen_cuda_dev_state_step(const zen_cuda_linear_layer* l, int rule, const float* d_proj, const int* d_pos, float* d_out, void* stream) {
    ZC_ENTER(stream, linear_ok(l, rule) && d_proj && d_pos && d_out, "state_step");
    const zk::LinearLayer d = device_form(*l, rule);
    const bool small = d.pitch <= 128;
    auto go = [&](auto kernel, size_t smem) { return launch(e, kernel, dim3(l->heads), dim3(zk::step_threads(small ? 4 : 8)), smem, d, d_proj, d_pos, d_out); };
    const size_t low = zk::step_low_floats(d) * sizeof(float);
    auto by_size = [&](auto which) {
        constexpr int kRule = decltype(which)::value;
        return small ? go(zk::state_step_kernel<kRule, 4>, low) : go(zk::state_step_kernel<kRule, 8>, low);
    };
    const cudaError_t r = rule == ZEN_CUDA_STATE_DELTA_RULE      ? by_size(std::integral_constant<int, zk::kDeltaRule>{})
                          : rule == ZEN_CUDA_STATE_DECAYED_WRITE ? by_size(std::integral_constant<int, zk::kDecayedWrite>{})
                                                                 : by_size(std::integral_constant<int, zk::kGatedWrite>{});
    return e.leave(r, "state_step");
}

int zen_cuda_dev_delta_inputs_rows(const zen_cuda_linear_layer* l, const float* d_proj, size_t ld, const float* d_decay, size_t decay_ld, size_t tokens, const int* d_pos,
                                   float* d_q, float* d_k, float* d_g, float* d_v, float* d_beta, void* stream) {
    ZC_ENTER(stream, linear_ok(l, ZEN_CUDA_STATE_DELTA_RULE) && d_proj && d_decay && decay_ld >= size_t(l->heads) * l->dim && tokens && tokens <= 0x7fffffffu && d_pos && d_q && d_k && d_g && d_v &&
                         d_beta, "delta_inputs_rows");
    const zk::LinearLayer d = device_form(*l, ZEN_CUDA_STATE_DELTA_RULE);
    const uint32_t items = 2 * l->kv_heads + (l->heads * l->vdim + 31) / 32 + l->heads, share = std::max(1u, std::min(64u, (items + 15) / 16));
    const cudaError_t r = launch(e, zk::delta_inputs_rows_kernel, dim3(u32((tokens + zk::kStrip - 1) / zk::kStrip), share), dim3(256), 0, d, d_proj, u32(ld), u32(tokens),
                                 d_decay, u32(decay_ld), d_pos, d_q, d_k, d_g, d_v, d_beta);
    if (!e.leave(r, "delta_inputs_rows")) return 0;
    return e.leave(launch(e, zk::conv_ring_update_kernel, dim3((d.conv.channels + 255) / 256), dim3(256), 0, d.conv, d_proj, u32(ld), u32(tokens), d_pos),
                   "delta_inputs_rows: ring");
}

int zen_cuda_dev_gated_write_inputs_rows(const zen_cuda_linear_layer* l, const float* d_proj, size_t ld, size_t tokens, float* d_q, float* d_f, void* stream) {
    ZC_ENTER(stream, linear_ok(l, ZEN_CUDA_STATE_GATED_WRITE) && d_proj && tokens && tokens <= 0x7fffffffu && d_q && d_f, "gated_write_inputs_rows");
    return e.leave(launch(e, zk::gated_write_inputs_rows_kernel, dim3(u32(tokens)), dim3(256), 0, device_form(*l, ZEN_CUDA_STATE_GATED_WRITE), d_proj, u32(ld), d_q, d_f), "gated_write_inputs_rows");
}

size_t zen_cuda_state_scan_workspace_bytes(const zen_cuda_linear_layer* l, int rule, size_t tokens) {
    if (!l) return 0;
    return (tokens + zk::kGroup - 1) / zk::kGroup * l->heads * zk::scan_record_floats(pitch32(l->dim), rule == ZEN_CUDA_STATE_DELTA_RULE) * sizeof(float);
}

int zen_cuda_dev_state_scan(const zen_cuda_linear_layer* l, int rule, const float* d_q, const float* d_k, const float* d_g, const float* d_v, size_t v_ld, const float* d_beta,
                            size_t tokens, void* d_workspace, size_t workspace_bytes, float* d_out, void* stream) {
    const bool delta = rule == ZEN_CUDA_STATE_DELTA_RULE;
    ZC_ENTER(stream, linear_ok(l, rule) && rule != ZEN_CUDA_STATE_DECAYED_WRITE && d_q && d_g && d_v && v_ld >= size_t(l->heads) * l->vdim && d_out && tokens &&
                         tokens <= 0x7fffffffu && l->heads <= 65535 && (!delta || (d_k && d_beta)) && d_workspace && !(reinterpret_cast<uintptr_t>(d_workspace) & 15) &&
                         workspace_bytes >= zen_cuda_state_scan_workspace_bytes(l, rule, tokens), "state_scan");
    zk::ScanParams p{};
    p.q = d_q; p.k = d_k; p.g = d_g; p.v = d_v; p.beta = d_beta; p.records = static_cast<float*>(d_workspace); p.state = l->state; p.out = d_out;
    p.tokens = u32(tokens); p.heads = l->heads; p.q_heads = delta ? l->kv_heads : l->heads; p.vdim = l->vdim; p.v_ld = u32(v_ld);
    return e.leave(run_scan(e, rule, l->dim, p, device_form(*l, rule)), "state_scan");
}

int zen_cuda_dev_decayed_write_scan(const zen_cuda_linear_layer* l, const float* d_proj, size_t ld, size_t tokens, const int* d_pos, void* d_workspace,
                                    size_t workspace_bytes, float* d_out, void* stream) {
    constexpr int rule = ZEN_CUDA_STATE_DECAYED_WRITE;
    ZC_ENTER(stream, linear_ok(l, rule) && d_proj && tokens && tokens <= 0x7fffffffu && l->heads <= 65535 && d_pos && d_out && d_workspace &&
                         !(reinterpret_cast<uintptr_t>(d_workspace) & 15) && workspace_bytes >= zen_cuda_state_scan_workspace_bytes(l, rule, tokens) &&
                         ld >= 2 * size_t(l->heads) * (l->dim + l->vdim) + (l->decay ? 0 : l->a2->cols), "decayed_write_scan");
    const size_t nq = size_t(l->heads) * l->dim, nv = size_t(l->heads) * l->vdim;
    zk::ScanParams p{};
    p.q = d_proj; p.k = d_proj + nq; p.v = d_proj + 2 * nq; p.low = d_proj + 2 * nq + 2 * nv; p.pos = d_pos;
    p.records = static_cast<float*>(d_workspace); p.state = l->state; p.out = d_out;
    p.tokens = u32(tokens); p.heads = p.q_heads = l->heads; p.vdim = l->vdim; p.v_ld = u32(ld);
    return e.leave(run_scan(e, rule, l->dim, p, device_form(*l, rule)), "decayed_write_scan");
}

}  // extern "C"
