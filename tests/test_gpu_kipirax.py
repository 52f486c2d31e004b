"""Kipirax on the GPU: every kernel alone against the plain float64 implementation (oracle/kipirax.py), then whole models in prompts,
portions, token by token and through generate()."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import kipirax_cases as cases
from dense_helpers import bf16_matrix, close, dev, feed_in, host, zeros
from oracle import kipirax as ref
from zeninfer_b200 import blocks, safetensors
from zeninfer_b200.backend import (DELTA_RULE, DENSE_PLAIN, DENSE_SOFTCAP, DENSE_SQUARED_RELU, GATED_WRITE, BackendError, LinearLayer, SublayerEnd, WindowAttention)
from zeninfer_b200.dense_decoder import round_up
from zeninfer_b200.kipirax import KipiraxDecoder, delta_rows

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_BAR, BF16_BAR = 5e-5, 4e-2       # logit_error of a whole model in either precision


@pytest.fixture(scope="module")
def be():
    from zeninfer_b200 import Backend
    return Backend()


ACTS = {DENSE_PLAIN: lambda z, cap: z, DENSE_SQUARED_RELU: lambda z, cap: np.maximum(z, 0) ** 2, DENSE_SOFTCAP: lambda z, cap: cap * np.tanh(z / cap)}


# ---- products ----
@pytest.mark.parametrize("rows,cols", [(1, 1), (7, 20), (149, 300), (1000, 256), (130, 4104), (33, 9000), (2500, 72)])
@pytest.mark.parametrize("act", [DENSE_PLAIN, DENSE_SQUARED_RELU, DENSE_SOFTCAP])
def test_dense_gemv(be, rows, cols, act):
    h, w = bf16_matrix(be, rows, cols, rows + cols)
    x = np.random.default_rng(3).standard_normal(cols).astype(np.float32) * np.float32(2.0)
    dx, y = dev(x), zeros(rows + 3)
    be.dev_dense_gemv([(h, dx.data_ptr(), y.data_ptr())], act=act, cap=1.5)
    got = host(y)
    close(got[:rows], ACTS[act](w @ x, 1.5))
    assert not got[rows:].any()
    be.dev_free(h)


def test_dense_gemv_several_tasks(be):
    shapes = [(70, 40), (333, 1100), (5, 256), (201, 8)]
    mats = [bf16_matrix(be, r, c, i) for i, (r, c) in enumerate(shapes)]
    xs = [dev(np.random.default_rng(i).standard_normal(c)) for i, (_, c) in enumerate(shapes)]
    ys = [zeros(r) for r, _ in shapes]
    be.dev_dense_gemv([(m[0], x.data_ptr(), y.data_ptr()) for m, x, y in zip(mats, xs, ys)])
    for m, x, y in zip(mats, xs, ys):
        close(host(y), m[1] @ host(x))
        be.dev_free(m[0])


@pytest.mark.parametrize("rows,cols,tokens", [(1, 8, 2), (130, 64, 33), (300, 90, 129), (257, 1000, 7), (1024, 520, 257), (96, 24, 512), (4100, 70, 20), (20000, 40, 300)])
@pytest.mark.parametrize("exact", [False, True])
def test_dense_gemm(be, rows, cols, tokens, exact):
    import torch
    h, w = bf16_matrix(be, rows, cols, rows)
    ld, out_ld = round_up(cols, 8), rows + 5
    x = torch.full((tokens, ld), 7.0, device="cuda")             # columns past the real ones must not count
    x[:, :cols] = dev(np.random.default_rng(4).standard_normal((tokens, cols)))
    if not exact:
        x = x.to(torch.bfloat16)
    want = host(x)[:, :cols].astype(np.float64) @ w.T
    for act in (DENSE_PLAIN, DENSE_SQUARED_RELU, DENSE_SOFTCAP):
        out = zeros(tokens, out_ld)
        be.dev_dense_gemm(h, x.data_ptr(), ld, tokens, out.data_ptr(), out_ld, exact=exact, act=act, cap=1.25)
        got = host(out)
        close(got[:, :rows], ACTS[act](want, 1.25))
        assert not got[:, rows:].any()
    if not exact:
        out = torch.zeros((tokens, out_ld), dtype=torch.bfloat16, device="cuda")
        be.dev_dense_gemm(h, x.data_ptr(), ld, tokens, out.data_ptr(), out_ld, out_bf16=True, act=DENSE_SQUARED_RELU)
        close(host(out)[:, :rows], np.maximum(want, 0) ** 2, 6e-3)
    be.dev_check(0)
    be.dev_free(h)


def test_products_refuse_bad_arguments(be):
    h, _ = bf16_matrix(be, 16, 24, 0)
    y = zeros(64)
    with pytest.raises(BackendError):
        be.dev_dense_gemm(h, y.data_ptr() + 4, 24, 2, y.data_ptr(), 16)          # bf16 rows must be 16-byte aligned
    with pytest.raises(BackendError):
        be.dev_dense_gemm(h, y.data_ptr(), 20, 2, y.data_ptr(), 16)              # pitch below the columns
    with pytest.raises(BackendError):
        be.dev_dense_gemv([(h, None, y.data_ptr())])
    with pytest.raises(BackendError):
        be.dev_gemv([h], [y.data_ptr()], y.data_ptr(), 1, 1)                     # the quantised product does not take a bf16 matrix
    be.dev_free(h)


# ---- the end of a sublayer ----
def sublayer_case(n, T, groups, two, view, seed=0):
    rng = np.random.default_rng(seed)
    vec = lambda: (1 + 0.3 * rng.standard_normal(n)).astype(np.float32)
    a = dict(x=rng.standard_normal((T, n)).astype(np.float32), ya=2 * rng.standard_normal((T, n)).astype(np.float32), yb=0.1 * rng.standard_normal((T, n)).astype(np.float32),
             wa=vec(), wb=vec(), norm=vec(), shift=rng.random(n).astype(np.float32), before=rng.standard_normal(n).astype(np.float32), out=vec())
    eps = 1e-3
    y = a["ya"].astype(np.float64)
    if two:
        y = 0.5 * (ref.rms(y, eps) * a["wa"] + ref.rms(a["yb"].astype(np.float64), eps) * a["wb"])
    x = a["x"] + ref.grouped_rms_norm(y, a["norm"], groups, eps)
    if view == "shift":
        seen = x + (np.concatenate([a["before"][None], x[:-1]]) - x) * a["shift"]
    else:
        seen = ref.grouped_rms_norm(x, a["out"], groups, eps) if view == "norm" else x
    d = {k: dev(v) for k, v in a.items()}
    x_out, keep = zeros(T, n), zeros(n)
    P = lambda t: t.data_ptr()
    end = SublayerEnd(P(d["x"]), P(x_out), P(d["ya"]), P(d["yb"]) if two else None, P(d["wa"]), P(d["wb"]), P(d["norm"]), P(keep), P(d["shift"]) if view == "shift" else None,
                      P(d["before"]) if view == "shift" else None, P(d["out"]) if view == "norm" else None, n, groups, eps)
    return a, d, end, x_out, keep, x, seen


@pytest.mark.parametrize("n,T,groups", [(90, 5, 3), (256, 1, 1), (1000, 37, 8), (64, 3, 64), (4096, 9, 4)])
@pytest.mark.parametrize("two", [False, True])
@pytest.mark.parametrize("view", ["plain", "shift", "norm"])
def test_sublayer_end(be, n, T, groups, two, view):
    import torch
    a, d, end, x_out, keep, x, seen = sublayer_case(n, T, groups, two, view)
    ld = round_up(n, 8)
    for bf16 in (False, True):
        out = torch.full((T, ld), 5.0, dtype=torch.bfloat16 if bf16 else torch.float32, device="cuda")
        be.dev_sublayer_end_rows(end, T, out.data_ptr(), ld, bf16)
        got = host(out)
        close(got[:, :n], seen, 6e-3 if bf16 else 2e-5)
        assert not got[:, n:].any()
    close(host(x_out), x)
    assert np.array_equal(host(keep), a["x"][-1])
    if T == 1:                                   # the same inside a decode product
        h, w = bf16_matrix(be, 77, n, 9)
        x_out.zero_(), keep.zero_()
        y = zeros(77)
        be.dev_dense_gemv([(h, None, y.data_ptr())], pre=end)
        close(host(y), w @ seen[0])
        close(host(x_out), x)
        assert np.array_equal(host(keep), a["x"][-1])
        be.dev_free(h)


def test_embedding_rows(be):
    import torch
    c, _, bits, w = cases.model("ragged")
    e, p = (be.dev_upload("BF16", bits[n].view(np.uint8), *bits[n].shape) for n in ("embed", "pos"))
    ids, pos, out = dev([5, 0, 202, 5], np.int64), dev([637], np.int32), zeros(4, 90)
    be.dev_embed_rows_bf16(e, p, ids.data_ptr(), 3, pos.data_ptr(), out.data_ptr())
    assert np.array_equal(host(out)[:3], w["embed"][[5, 0, 202]] + w["pos"][637:640])
    be.dev_embed_rows_bf16(e, None, ids.data_ptr(), 4, None, out.data_ptr())
    assert np.array_equal(host(out), w["embed"][[5, 0, 202, 5]])
    be.dev_check(0)
    be.dev_embed_rows_bf16(e, p, ids.data_ptr(), 4, pos.data_ptr(), out.data_ptr())          # position 640 is past the table
    torch.cuda.synchronize()
    with pytest.raises(BackendError, match="position"):
        be.dev_check(0)
    bad = dev([203], np.int64)
    be.dev_embed_rows_bf16(e, None, bad.data_ptr(), 1, None, out.data_ptr())
    with pytest.raises(BackendError, match="token"):
        be.dev_check(0)
    be.dev_free(e), be.dev_free(p)


# ---- windowed attention ----
WINDOWS = [  # heads, kv_heads, dim, vdim, window, keep_first
    (4, 2, 24, 20, 16, 3), (3, 1, 50, 70, 33, 0), (8, 2, 32, 32, 64, 1), (2, 2, 136, 40, 20, 37), (4, 1, 96, 96, 96, 5), (6, 2, 100, 160, 1, 2), (2, 1, 200, 256, 700, 4),
]


@pytest.mark.parametrize("heads,kv,dim,vdim,window,keep", WINDOWS)
def test_window_attention(be, heads, kv, dim, vdim, window, keep):
    """A prompt in portions and decoded tokens, against keys that decide the output wherever they are visible: at the last kept and
    the first dropped position, across block borders, and so placed that the last tokens pass their window's edge."""
    T, eps = 180, 1e-5
    planted = sorted({j for j in (keep - 1, keep, 31, 32, 60, 100, T - 24 - window) if 0 <= j < T})
    q, k, v, qw, kw = cases.standout_attention(T, heads, kv, dim, vdim, planted, window)
    scale = 40.0 / dim
    qn, kn = ref.rms(q.astype(np.float64), eps) * qw, ref.rms(k.astype(np.float64), eps) * kw
    want = ref.window_attention(qn, kn, v.astype(np.float64), scale, window, keep)
    gates = np.random.default_rng(7).standard_normal((T, heads)).astype(np.float32)
    row = heads * dim + kv * dim + kv * vdim
    proj = dev(np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], axis=1))
    pitch = round_up(max(dim, vdim), 32)
    for cuts in ([T - 40], [2, 3, 50, 1, 17, T - 120], [33, 64, 2, 30]):
        kc, vc, qb, out = zeros(T, kv, pitch), zeros(T, kv, pitch), zeros(T, heads, pitch), zeros(T, heads, pitch)
        dq, dk = dev(qw), dev(kw)
        a = WindowAttention(heads, kv, dim, vdim, pitch, window, keep, 1, T, scale, eps, dq.data_ptr(), dk.data_ptr(), kc.data_ptr(), vc.data_ptr())
        pos, done, got = dev([0], np.int32), 0, np.zeros_like(want)
        at = lambda t, col: proj.data_ptr() + 4 * (t * row + col)
        for n in cuts:
            be.dev_window_attention_rows(a, at(done, 0), at(done, heads * dim), at(done, (heads + kv) * dim), row, n, pos.data_ptr(), qb.data_ptr(), out.data_ptr())
            got[done:done + n] = host(out)[:n, :, :vdim]
            done += n
            pos.fill_(done)
        prompt = done
        one, g = zeros(heads, vdim), dev(gates)
        while done < T:
            be.dev_window_attention_step(a, at(done, 0), at(done, heads * dim), at(done, (heads + kv) * dim), g[done].data_ptr(), pos.data_ptr(), one.data_ptr())
            got[done] = host(one)
            done += 1
            pos.fill_(done)
        be.dev_check(0)
        close(got[:prompt], want[:prompt], 1e-4)
        close(got[prompt:], (want * ref.sigmoid(gates.astype(np.float64))[:, :, None])[prompt:], 1e-4)


def test_attention_reports_a_position_past_the_cache(be):
    heads, kv, dim, vdim, T = 2, 1, 8, 8, 4
    kc, vc, out, w = zeros(T, kv, 32), zeros(T, kv, 32), zeros(8, heads, 32), dev(np.ones(dim))
    a = WindowAttention(heads, kv, dim, vdim, 32, 4, 0, 1, T, 0.3, 1e-5, w.data_ptr(), w.data_ptr(), kc.data_ptr(), vc.data_ptr())
    proj, pos, qb = zeros(8, 64), dev([T], np.int32), zeros(8, heads, 32)
    be.dev_window_attention_step(a, proj.data_ptr(), proj.data_ptr(), proj.data_ptr(), None, pos.data_ptr(), out.data_ptr())
    with pytest.raises(BackendError, match="position"):
        be.dev_check(0)
    pos.fill_(2)
    be.dev_window_attention_rows(a, proj.data_ptr(), proj.data_ptr(), proj.data_ptr(), 64, 3, pos.data_ptr(), qb.data_ptr(), out.data_ptr())
    with pytest.raises(BackendError, match="position"):
        be.dev_check(0)


# ---- mixers with a matrix state ----
RULES = {"delta": DELTA_RULE, "write": GATED_WRITE}
CUTS = [[75], [2, 3, 40, 7, 9], [1, 8, 16, 17], [33]]


def linear_case(be, kind, seed, **m):
    """A layer on the device, its projection rows for T tokens, and the oracle's outputs before the output projection."""
    rng = np.random.default_rng(seed)
    T, eps, f32 = 84, 1e-5, np.float32
    keep, h = {}, m["heads"]
    keep["norm"] = (1 + 0.2 * rng.standard_normal(m["vdim"])).astype(f32)
    keep["state"] = np.zeros((h, m["vdim"], round_up(m["dim"], 32)), f32)
    if kind == "delta":
        cfg = type("M", (), m)
        rows = delta_rows(cfg, m["rank_a"], m["rank_g"])
        nq, nv = m["kv_heads"] * m["dim"], h * m["vdim"]
        conv = rng.standard_normal((2 * nq + nv, m["conv"])).astype(f32)
        keep.update(conv=conv.T.copy(), a_log=rng.uniform(-1, 1.5, h).astype(f32), dt_bias=(rng.standard_normal(h * m["dim"]) - 3).astype(f32),
                    ring=np.full((m["conv"], 2 * nq + nv), 99.0, f32))
        a2, wa2 = bf16_matrix(be, h * m["dim"], m["rank_a"], seed + 1)
        g2, wg2 = bf16_matrix(be, h * m["vdim"], m["rank_g"], seed + 2)
        w = {**cases.selectors(rows), "q.conv": conv[:nq], "k.conv": conv[nq:2 * nq], "v.conv": conv[2 * nq:], "A_log": keep["a_log"], "dt_bias": keep["dt_bias"],
             "a2": wa2, "g2": wg2, "norm": keep["norm"], "o": np.eye(nv)}
    else:
        n = h * m["dim"]
        rows = [("q", n), ("f", n), ("v", h * m["vdim"])]
        keep.update(f_bias=rng.standard_normal(n).astype(f32), lower=rng.uniform(0, 0.95, n).astype(f32))
        w = {**cases.selectors(rows), "f.b": keep["f_bias"], "lower": keep["lower"], "norm": keep["norm"], "o": np.eye(h * m["vdim"])}
    proj = rng.standard_normal((T, sum(n for _, n in rows))).astype(f32)
    want = (ref.channel_delta if kind == "delta" else ref.parallel_right)(proj.astype(np.float64), w, m, eps)
    d = {n: dev(t) for n, t in keep.items()}
    extra = dict(a2=a2, g2=g2) if kind == "delta" else {}
    layer = LinearLayer(h, m.get("kv_heads", h), m["dim"], m["vdim"], m.get("conv", 0), eps, **extra, **{n: t.data_ptr() for n, t in d.items()})
    return T, rows, proj, want, d, layer, extra


def run_linear(be, kind, m, case, cuts):
    T, rows, proj, want, d, layer, extra = case
    h, dim, vdim, g = m["heads"], m["dim"], m["vdim"], m.get("kv_heads", m["heads"])
    pitch, N = round_up(dim, 32), proj.shape[1]
    P = lambda t: t.data_ptr()
    dp, pos, got, done = dev(proj), dev([0], np.int32), np.zeros_like(want), 0
    ws = zeros(be.state_scan_workspace_bytes(layer, RULES[kind], T) // 4)
    q, k, gd, v, beta, o = zeros(T, g, pitch), zeros(T, g, pitch), zeros(T, h, pitch), zeros(T, h * vdim), zeros(T, h), zeros(T, h, vdim)
    y, at = zeros(T, h * vdim), {}
    col = 0
    for n, r in rows:
        at[n] = col
        col += r
    for n in cuts:
        row = dp[done:]
        if kind == "delta":
            decay, gate = zeros(T, h * dim), zeros(T, h * vdim)
            be.dev_dense_gemm(extra["a2"], P(row) + 4 * at["a1"], N, n, P(decay), h * dim, exact=True)
            be.dev_dense_gemm(extra["g2"], P(row) + 4 * at["g1"], N, n, P(gate), h * vdim, exact=True)
            be.dev_delta_inputs_rows(layer, P(row), N, P(decay), h * dim, n, P(pos), P(q), P(k), P(gd), P(v), P(beta))
            be.dev_state_scan(layer, DELTA_RULE, P(q), P(k), P(gd), P(v), h * vdim, P(beta), n, P(ws), 4 * ws.numel(), P(o))
            be.dev_head_outputs_rows(P(o), n, h, vdim, vdim, P(y), h * vdim, False, weight=layer.norm, eps=layer.eps, gate=P(gate), gate_ld=h * vdim, gate_mode=2)
        else:
            be.dev_gated_write_inputs_rows(layer, P(row), N, n, P(q), P(gd))
            be.dev_state_scan(layer, GATED_WRITE, P(q), None, P(gd), P(row) + 4 * at["v"], N, None, n, P(ws), 4 * ws.numel(), P(o))
            be.dev_head_outputs_rows(P(o), n, h, vdim, vdim, P(y), h * vdim, False, weight=layer.norm, eps=layer.eps)
        got[done:done + n] = host(y)[:n]
        done += n
        pos.fill_(done)
    one = zeros(h * vdim)
    while done < T:
        be.dev_state_step(layer, RULES[kind], P(dp[done]), P(pos), P(one))
        got[done] = host(one)
        done += 1
        pos.fill_(done)
    be.dev_check(0)
    return got


@pytest.mark.parametrize("m", [dict(heads=4, kv_heads=2, dim=20, vdim=28, conv=3, rank_a=10, rank_g=7), dict(heads=3, kv_heads=1, dim=64, vdim=33, conv=1, rank_a=8, rank_g=70),
                               dict(heads=2, kv_heads=2, dim=130, vdim=65, conv=6, rank_a=140, rank_g=3), dict(heads=1, kv_heads=1, dim=256, vdim=256, conv=4, rank_a=16, rank_g=300), dict(heads=2, kv_heads=1, dim=18, vdim=40, conv=11, rank_a=5, rank_g=9),
                               dict(heads=2, kv_heads=2, dim=32, vdim=32, conv=8, rank_a=64, rank_g=64)])
@pytest.mark.parametrize("cuts", CUTS)
def test_delta_rule(be, m, cuts):
    case = linear_case(be, "delta", m["dim"], **m)
    close(run_linear(be, "delta", m, case, cuts), case[3], 1e-4)
    for hnd in case[6].values():
        be.dev_free(hnd)


@pytest.mark.parametrize("m", [dict(heads=3, dim=12, vdim=37), dict(heads=4, dim=96, vdim=20), dict(heads=1, dim=256, vdim=200), dict(heads=2, dim=33, vdim=256)])
@pytest.mark.parametrize("cuts", CUTS)
def test_gated_write(be, m, cuts):
    case = linear_case(be, "write", m["dim"], **m)
    close(run_linear(be, "write", m, case, cuts), case[3], 1e-4)


def test_scan_keeps_a_write_far_away(be):
    # one token writes, nothing decays and nothing else matches it: five hundred tokens later the read-out is still exact
    h, dim, vdim, T = 2, 40, 24, 520
    rng = np.random.default_rng(0)
    k = np.zeros((T, h, 64), np.float32)
    k[:, :, 1:40] = rng.standard_normal((T, h, 39))
    k /= np.sqrt((k ** 2).sum(-1, keepdims=True))
    k[3], k[3, :, 0] = 0.0, 1.0
    q = k.copy()
    q[-1] = k[3]
    v, beta, g = rng.standard_normal((T, h, vdim)).astype(np.float32), np.ones((T, h), np.float32), np.ones((T, h, 64), np.float32)
    norm, state, out, dummy = dev(np.ones(vdim)), zeros(h, vdim, 64), zeros(T, h, vdim), zeros(h * dim * 8)
    a2, _ = bf16_matrix(be, h * dim, 4, 0)
    g2, _ = bf16_matrix(be, h * vdim, 4, 0)
    P = lambda t: t.data_ptr()
    layer = LinearLayer(h, h, dim, vdim, 1, 1e-5, conv=P(dummy), a_log=P(dummy), dt_bias=P(dummy), a2=a2, g2=g2, norm=P(norm), ring=P(dummy), state=P(state))
    d = [dev(t) for t in (q, k, g, v, beta)]
    ws = zeros(be.state_scan_workspace_bytes(layer, DELTA_RULE, T) // 4)
    be.dev_state_scan(layer, DELTA_RULE, P(d[0]), P(d[1]), P(d[2]), P(d[3]), h * vdim, P(d[4]), T, P(ws), 4 * ws.numel(), P(out))
    with pytest.raises(BackendError):
        be.dev_state_scan(layer, DELTA_RULE, P(d[0]), P(d[1]), P(d[2]), P(d[3]), h * vdim, P(d[4]), T, P(ws), 4 * ws.numel() - 4, P(out))
    close(host(out)[-1], v[3], 1e-4)
    be.dev_free(a2), be.dev_free(g2)


@pytest.mark.parametrize("heads,width,pitch,mode", [(3, 37, 37, 0), (4, 50, 64, 1), (2, 200, 200, 2), (40, 5, 32, 1)])
def test_head_outputs(be, heads, width, pitch, mode):
    rng = np.random.default_rng(heads)
    T, ld = 6, round_up(heads * width, 8) + 8
    o, w = rng.standard_normal((T, heads, pitch)).astype(np.float32), (1 + 0.2 * rng.standard_normal(width)).astype(np.float32)
    gate = rng.standard_normal((T, 11 + (heads if mode == 1 else heads * width))).astype(np.float32)
    for weight in (None, w):
        want = o[:, :, :width].astype(np.float64)
        if weight is not None:
            want = ref.rms(want, 1e-4) * w
        if mode:
            gv = ref.sigmoid(gate[:, 11:].astype(np.float64))
            want = want * (gv[:, :, None] if mode == 1 else gv.reshape(T, heads, width))
        do, dw, dg, out = dev(o), dev(w), dev(gate), zeros(T, ld)
        be.dev_head_outputs_rows(do.data_ptr(), T, heads, width, pitch, out.data_ptr(), ld, False, weight=dw.data_ptr() if weight is not None else None, eps=1e-4,
                                 gate=dg.data_ptr() + 44, gate_ld=gate.shape[1], gate_mode=mode)
        got = host(out)
        close(got[:, :heads * width], want.reshape(T, -1))
        assert not got[:, heads * width:].any()


# ---- whole models ----
def decoder(be, name, dtype="float32", chunk=None, **kw):
    c, cfg, bits, weights = cases.model(name)
    dec = KipiraxDecoder(be, cfg, bits.__getitem__, dtype=dtype, **kw)
    if chunk:
        dec.PREFILL_CHUNK = chunk
    dec.capture()
    return c, weights, dec


@pytest.mark.parametrize("name", sorted(cases.CASES))
@pytest.mark.parametrize("dtype,bar", [("float32", F32_BAR), ("bfloat16", BF16_BAR)])
def test_model_prompts_portions_and_tokens(be, name, dtype, bar):
    c, weights, dec = decoder(be, name, dtype, chunk=64)
    ids = cases.tokens_for(c, 150)
    want, after = ref.forward(c, weights, ids)
    for cuts in ([150], [1], [2], [97, 1, 2, 3, 33, 1], [64, 64, 1], [5, 1, 1, 30]):
        assert cases.logit_error(feed_in(dec, ids, cuts), want) <= bar, cuts
    # the residual stream after the last layer, of the last block fed
    dec.reset()
    dec.feed(ids[:100])
    dec.feed(ids[100:150])
    close(host(dec._prefill_buffers()["last"])[:50], after[-1][100:], 1e-4 if dtype == "float32" else 5e-2)
    # one token alone, and two
    for n in (1, 2):
        dec.reset()
        assert cases.logit_error(dec.feed(ids[:n], list(range(n))), want[:n]) <= bar
    dec.close()


def test_a_sequence_leaves_nothing_behind(be):
    c, weights, dec = decoder(be, "ragged", chunk=64)
    a, b = cases.tokens_for(c, 120, 5), cases.tokens_for(c, 61, 6)
    first = feed_in(dec, b, [40, 1, 20])
    for _ in range(2):
        feed_in(dec, a, [64, 3, 1])                              # a longer sequence fills cache, ring and states
        assert np.array_equal(feed_in(dec, b, [40, 1, 20]), first)
    dec.generate(a[:30], 20)
    assert np.array_equal(feed_in(dec, b, [40, 1, 20]), first)
    assert cases.logit_error(first, ref.forward(c, weights, b)[0]) <= F32_BAR
    dec.close()


def test_wanted_places(be):
    c, _, dec = decoder(be, "last_bare", chunk=32)
    ids = cases.tokens_for(c, 70)
    every = feed_in(dec, ids, [70])
    dec.reset()
    picked = dec.feed(ids, [69, 0, 31, 32, 31])                  # any order, block edges, one of them twice
    assert np.array_equal(picked, every[[69, 0, 31, 32, 31]])
    dec.reset()
    assert dec.feed(ids[:9]).shape == (0, c["vocab"])
    for bad in (lambda: dec.feed([1], [1]), lambda: dec.feed([c["vocab"]]), lambda: dec.feed([-1]), lambda: dec.feed([0] * 640)):
        with pytest.raises(ValueError):
            bad()
    dec.close()


def test_long_decoding(be):
    c, weights, dec = decoder(be, "ragged")
    ids = cases.tokens_for(c, 420, 9)
    want, _ = ref.forward(c, weights, ids)
    got = feed_in(dec, ids, [20, 1])
    assert cases.logit_error(got, want) <= 2 * F32_BAR
    dec.close()


def test_cache_of_just_the_right_size(be):
    c, weights, dec = decoder(be, "wide", max_positions=50)
    ids = cases.tokens_for(c, 50)
    assert cases.logit_error(feed_in(dec, ids, [49, 1]), ref.forward(c, weights, ids)[0]) <= F32_BAR
    with pytest.raises(ValueError):
        dec.feed(ids[:1])
    dec.close()


@pytest.mark.parametrize("name", ["ragged", "last_bare"])
def test_generate(be, name):
    c, weights, dec = decoder(be, name, chunk=32)
    prompt = cases.tokens_for(c, 41, 3)
    for p in (prompt, prompt[:1]):
        ids = dec.generate(p, 24)
        logits, _ = ref.forward(c, weights, p + ids)
        for i, tok in enumerate(ids):
            row = logits[len(p) - 1 + i]
            assert row.max() - row[tok] <= 1e-3 * np.abs(row).max()          # the oracle's maximum, but for a tie within rounding
        assert dec.generate(p, 24) == ids
        assert dec.generate(p, 24, batched_prefill=False) == ids
        assert dec.generate(p, 24, temperature=0.7, top_k=1, seed=4) == ids  # one candidate: sampling has no choice
    drawn = dec.generate(prompt, 24, temperature=1.5, seed=1)
    assert drawn == dec.generate(prompt, 24, temperature=1.5, seed=1) and all(0 <= t < c["vocab"] for t in drawn)
    with pytest.raises(ValueError):
        dec.generate(prompt, 640)
    dec.close()


def test_missing_and_misshapen_tensors_are_refused(be):
    c, cfg, bits, _ = cases.model("last_bare")
    with pytest.raises(KeyError):
        KipiraxDecoder(be, cfg, {n: t for n, t in bits.items() if n != "l1.mix.right.lower"}.__getitem__)
    bad = {**bits, "l0.mix.o": bits["l0.mix.o"][:-1]}
    with pytest.raises(ValueError, match="l0.mix.o"):
        KipiraxDecoder(be, cfg, bad.__getitem__)


def test_commands(be, tmp_path):
    """bin/trace_run and the generate command on a model folder, each in a process of its own."""
    c, cfg, bits, weights = cases.model("ragged")
    (tmp_path / "config.json").write_text(json.dumps(c))
    safetensors.write(str(tmp_path / "model.safetensors"), bits)
    ids = cases.tokens_for(c, 60, 8)
    want, _ = ref.forward(c, weights, ids)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:50], "want": [0, 49]}], "end": []}, {"step": 1, "entries": [{"id": "a", "tokens": ids[50:58], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[58:], "want": [1]}], "end": ["a"]}, {"step": 3, "entries": [{"id": "b", "tokens": ids[:5], "want": [4]}], "end": ["b"]}]
    for dtype, bar in (("float32", F32_BAR), ("bfloat16", BF16_BAR)):
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "60"], text=True,
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"])
        assert cases.logit_error(np.concatenate([read(0), read(2), read(3)]), want[[0, 49, 59, 4]]) <= bar
        assert not (tmp_path / "1.f32").exists()
    run = lambda *a: subprocess.run([sys.executable, "-m", "zeninfer_b200", *a], cwd=ROOT, text=True, capture_output=True, timeout=300)
    r = run("generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt-ids", ",".join(map(str, ids)), "--max-new", "6")
    assert r.returncode == 0, r.stderr
    out = [int(t) for t in r.stdout.strip().split(",")]
    dec = KipiraxDecoder(be, cfg, bits.__getitem__, dtype="float32")
    dec.capture()
    assert out == dec.generate(ids, 6)
    dec.close()
    assert run("info", "--model", str(tmp_path)).stdout.strip() == "Kipirax"
    assert run("nonsense").returncode == 2


def test_llama_feeds_through_the_same_runtime(be):
    """The shared feed() on the llama decoder: portions against the whole, and against generate()'s picks."""
    from zeninfer_b200.backend import ACT_FP32
    from zeninfer_b200.llama import LlamaConfig, LlamaDecoder, synthetic_tensors
    cfg = LlamaConfig(embedding=256, layers=2, heads=4, kv_heads=2, head_dim=64, ffn=512, vocab=512, context=128)
    dec = LlamaDecoder(be, cfg, synthetic_tensors(cfg, 3), act_mode=ACT_FP32)
    dec.capture()
    ids = np.random.default_rng(0).integers(0, cfg.vocab, 70).tolist()
    whole, parts = feed_in(dec, ids, [70]), feed_in(dec, ids, [40, 1, 20])
    assert cases.logit_error(parts, whole) <= 2e-3
    assert dec.generate(ids, 1) == [int(whole[-1].argmax())]
    dec.close()
