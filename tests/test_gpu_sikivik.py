"""Sikivik on the GPU: what it adds to the kernels, each alone against the plain float64 implementation (oracle/sikivik.py), then whole
models in prompts, portions, token by token and through generate()."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import sikivik_cases as cases
from dense_helpers import bf16_matrix, close, dev, feed_in, host, zeros
from oracle import sikivik as ref
from zeninfer_b200 import blocks, safetensors
from zeninfer_b200.backend import DECAYED_WRITE, DENSE_SQUARED_RELU, BackendError, LinearLayer, SublayerEnd, WindowAttention
from zeninfer_b200.dense_decoder import round_up
from zeninfer_b200.sikivik import Rotation, SikivikDecoder, rotation_tables

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_BAR, BF16_BAR = 5e-5, 4e-2       # logit_error of a whole model in either precision
P = lambda t: None if t is None else t.data_ptr()


@pytest.fixture(scope="module")
def be():
    from zeninfer_b200 import Backend
    return Backend()


# ---- products with a bias and gated pairs of rows ----
SHAPES = [(2, 1, 8), (7, 2, 20), (301, 100, 300), (149, 0, 256), (600, 300, 72), (1501, 640, 4104), (131, 64, 90)]      # rows, pairs, columns


@pytest.mark.parametrize("rows,pairs,cols", SHAPES)
def test_gemv_pairs_and_bias(be, rows, pairs, cols):
    h, w = bf16_matrix(be, rows, cols, rows + cols)
    rng = np.random.default_rng(3)
    x, b = rng.standard_normal(cols).astype(np.float32) * 2, rng.standard_normal(rows - 2 * pairs + 1).astype(np.float32)
    dx, db, y, gated = dev(x), dev(b), zeros(rows - 2 * pairs + 3), zeros(pairs + 3)
    want = w @ x
    for act in (0, DENSE_SQUARED_RELU):
        be.dev_dense_gemv([(h, P(dx), P(y))], bias=P(db), gated=P(gated), gated_pairs=pairs, act=act)
        tail = want[2 * pairs:] + b[:-1]
        if rows > 2 * pairs:
            close(host(y)[:-3], np.maximum(tail, 0) ** 2 if act else tail)
        if pairs:
            close(host(gated)[:-3], ref.silu(want[0:2 * pairs:2]) * want[1:2 * pairs:2])
        assert not host(y)[rows - 2 * pairs:].any() and not host(gated)[pairs:].any()
    if pairs:
        with pytest.raises(BackendError):
            be.dev_dense_gemv([(h, P(dx), P(y))], gated_pairs=pairs)
        with pytest.raises(BackendError):
            be.dev_dense_gemv([(h, P(dx), P(y))], gated=P(gated), gated_pairs=rows // 2 + 1)
    be.dev_free(h)


@pytest.mark.parametrize("rows,pairs,cols", SHAPES)
@pytest.mark.parametrize("tokens", [2, 33, 257])
@pytest.mark.parametrize("exact", [False, True])
def test_gemm_pairs_and_bias(be, rows, pairs, cols, tokens, exact):
    import torch
    h, w = bf16_matrix(be, rows, cols, rows)
    rng = np.random.default_rng(4)
    ld, n = round_up(cols, 8), rows - 2 * pairs
    x = torch.full((tokens, ld), 7.0, device="cuda")
    x[:, :cols] = dev(rng.standard_normal((tokens, cols)))
    if not exact:
        x = x.to(torch.bfloat16)
    b = rng.standard_normal(n + 1).astype(np.float32)
    db, out = dev(b), zeros(tokens, n + 5)
    gated = torch.zeros((tokens, pairs + 3), dtype=torch.float32 if exact else torch.bfloat16, device="cuda")
    be.dev_dense_gemm(h, P(x), ld, tokens, P(out), n + 5, exact=exact, bias=P(db), gated=P(gated), gated_ld=pairs + 3, gated_pairs=pairs)
    want = host(x)[:, :cols].astype(np.float64) @ w.T
    got, g = host(out), host(gated)
    if n:
        close(got[:, :n], want[:, 2 * pairs:] + b[:-1])
    if pairs:
        close(g[:, :pairs], ref.silu(want[:, 0:2 * pairs:2]) * want[:, 1:2 * pairs:2], 2e-5 if exact else 6e-3)
    assert not got[:, n:].any() and not g[:, pairs:].any()
    be.dev_check(0)
    if pairs:
        with pytest.raises(BackendError):
            be.dev_dense_gemm(h, P(x), ld, tokens, P(out), n + 5, exact=exact, gated=P(gated), gated_ld=pairs - 1, gated_pairs=pairs)
    be.dev_free(h)


# ---- the residual add without a norm of its own ----
@pytest.mark.parametrize("n,T", [(90, 5), (256, 1), (1000, 37), (4096, 9)])
def test_plain_sublayer_end(be, n, T):
    import torch
    rng = np.random.default_rng(n)
    x, y, w = rng.standard_normal((T, n)).astype(np.float32), rng.standard_normal((T, n)).astype(np.float32), (1 + 0.3 * rng.standard_normal(n)).astype(np.float32)
    dx, dy, dw, x_out = dev(x), dev(y), dev(w), zeros(T, n)
    end = SublayerEnd(x_in=P(dx), x_out=P(x_out), y_a=P(dy), out_norm=P(dw), n=n, groups=1, eps=1e-4)
    want = ref.rms(x.astype(np.float64) + y, 1e-4) * w
    ld = round_up(n, 8)
    for bf16 in (False, True):
        out = torch.full((T, ld), 5.0, dtype=torch.bfloat16 if bf16 else torch.float32, device="cuda")
        be.dev_sublayer_end_rows(end, T, P(out), ld, bf16)
        close(host(out)[:, :n], want, 6e-3 if bf16 else 2e-5)
        assert not host(out)[:, n:].any() and np.array_equal(host(x_out), x + y)
    if T == 1:                                   # the same inside a decode product
        h, m = bf16_matrix(be, 77, n, 9)
        x_out.zero_()
        out = zeros(57)
        gated = zeros(10)
        be.dev_dense_gemv([(h, None, P(out))], pre=end, gated=P(gated), gated_pairs=10)
        prod = m @ want[0]
        close(host(out), prod[20:])
        close(host(gated), ref.silu(prod[0:20:2]) * prod[1:20:2])
        assert np.array_equal(host(x_out), x + y)
        be.dev_free(h)


@pytest.mark.parametrize("mode,gate", [(2, ref.sigmoid), (3, ref.silu)])
def test_head_outputs_beside_other_columns(be, mode, gate):
    rng = np.random.default_rng(mode)
    T, heads, width, pitch, ld = 6, 3, 37, 64, 150
    fill = round_up(heads * width, 8)
    o, g = rng.standard_normal((T, heads, pitch)).astype(np.float32), rng.standard_normal((T, 11 + heads * width)).astype(np.float32)
    do, dg, ones, out = dev(o), dev(g), dev(np.ones(width)), dev(np.full((T, ld), 9.0))
    be.dev_head_outputs_rows(P(do), T, heads, width, pitch, P(out), ld, False, weight=P(ones), eps=1e-3, gate=P(dg) + 44, gate_ld=g.shape[1], gate_mode=mode, fill=fill)
    want = ref.rms(o[:, :, :width].astype(np.float64), 1e-3).reshape(T, -1) * gate(g[:, 11:].astype(np.float64))
    got = host(out)
    close(got[:, :heads * width], want)
    assert not got[:, heads * width:fill].any() and (got[:, fill:] == 9.0).all()


# ---- attention with convolution, rotation and mixed values ----
WINDOWS = [  # heads, kv_heads, dim, vdim, window, taps, rotated dimensions
    (4, 2, 24, 20, 16, 3, 24), (3, 1, 50, 70, 33, 2, 18), (8, 2, 32, 32, 64, 4, 32), (2, 2, 136, 40, 20, 1, 70), (4, 1, 96, 96, 96, 6, 2), (6, 2, 100, 160, 1, 3, 100),
    (2, 1, 200, 256, 700, 5, 0), (4, 4, 48, 18, 2, 2, 46),
]


@pytest.mark.parametrize("heads,kv,dim,vdim,window,taps,rot", WINDOWS)
def test_rotary_window_attention(be, heads, kv, dim, vdim, window, taps, rot):
    """A prompt in portions and decoded tokens, against keys that decide the output wherever they are visible: across block borders,
    and so placed that prompt tokens and the last tokens pass their window's edge.  Values are kept, and mixed with others."""
    T = 180
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=20.0 / dim, mask=dict(size=window), conv=taps, rot=dict(base=300.0, dims=rot))
    planted = sorted({j for j in (31, 32, 60, 100, T - 24 - window, T - 60 - window) if 0 <= j < T})
    proj, conv = cases.standout_projections(T, m, planted, window)
    rows = [("q", heads * dim), ("k", kv * dim), ("v", kv * vdim), ("g", heads * vdim)]
    w = {**cases.selectors(rows), **{f"{n}.b": 0.0 for n in "qkvo"}, **{f"{n}.conv": t for n, t in zip("qkv", conv)}, "o": np.eye(heads * vdim), "vmix": 0.375}
    first = np.random.default_rng(1).standard_normal((T, kv, vdim)).astype(np.float32)
    N, channels, pitch = proj.shape[1], (heads + kv) * dim + kv * vdim, round_up(max(dim, vdim), 32)
    dp, dconv, dfirst = dev(proj), dev(np.concatenate(conv).T), dev(first)
    cos, sin = (dev(t) for t in rotation_tables(Rotation(300.0, rot), T))
    at = lambda t, col: P(dp) + 4 * (t * N + col)
    for cuts, mixes in (([T - 40], True), ([2, 3, 50, 1, 17, T - 120], False), ([33, 64, 2, 30], True)):
        want, values = ref.attention(proj.astype(np.float64), w, m, first.astype(np.float64) if mixes else None)
        kc, vc, qb, out, y = zeros(T, kv, pitch), zeros(T, kv, pitch), zeros(T, heads, pitch), zeros(T, heads, pitch), zeros(T, heads * vdim)
        ring, kept = dev(np.full((taps, channels), 99.0)), zeros(T, kv * vdim)
        a = WindowAttention(heads, kv, dim, vdim, pitch, window, 0, 0, T, m["scale"], 1e-5, k_cache=P(kc), v_cache=P(vc), rot_pairs=rot // 2, taps=taps, gate_values=1,
                            v_share=0.375, rot_cos=P(cos) if rot else None, rot_sin=P(sin) if rot else None, conv=P(dconv), ring=P(ring))
        pos, done, got = dev([0], np.int32), 0, np.zeros((T, heads * vdim))

        def values_at(t):
            a.v_first, a.v_keep = (P(dfirst) + 4 * t * kv * vdim if mixes else None), P(kept) + 4 * t * kv * vdim
        for n in cuts:
            values_at(done)
            be.dev_window_attention_rows(a, at(done, 0), at(done, heads * dim), at(done, (heads + kv) * dim), N, n, P(pos), P(qb), P(out))
            be.dev_head_outputs_rows(P(out), n, heads, vdim, pitch, P(y), heads * vdim, False, gate=at(done, channels), gate_ld=N, gate_mode=2)
            got[done:done + n] = host(y)[:n]
            done += n
            pos.fill_(done)
        one = zeros(heads, vdim)
        while done < T:
            values_at(done)
            be.dev_window_attention_step(a, at(done, 0), at(done, heads * dim), at(done, (heads + kv) * dim), at(done, channels), P(pos), P(one))
            got[done] = host(one).reshape(-1)
            done += 1
            pos.fill_(done)
        be.dev_check(0)
        close(got, want, 1e-4)
        close(host(kept).reshape(T, kv, vdim), values, 1e-4)


def test_rotary_attention_refuses_bad_arguments(be):
    kc, vc, out, t = zeros(4, 1, 32), zeros(4, 1, 32), zeros(8, 2, 32), zeros(1024)
    good = dict(k_cache=P(kc), v_cache=P(vc), rot_pairs=4, rot_cos=P(t), rot_sin=P(t), taps=2, conv=P(t), ring=P(t))
    pos = dev([2], np.int32)
    make = lambda **kw: WindowAttention(2, 1, 8, 8, 32, 4, 0, 0, 4, 0.3, 1e-5, **{**good, **kw})
    rows = lambda a, n, k=64: be.dev_window_attention_rows(a, P(t), P(t) + k, P(t) + 96, 32, n, P(pos), P(out), P(out))
    for bad in (make(rot_pairs=5), make(rot_cos=None), make(conv=None), make(q_weight=P(t)), make(q_weight=P(t), k_weight=P(t))):
        with pytest.raises(BackendError):
            rows(bad, 1)
        with pytest.raises(BackendError):
            be.dev_window_attention_step(bad, P(t), P(t), P(t), None, P(pos), P(out))
    with pytest.raises(BackendError, match="consecutive"):
        rows(make(), 1, 60)
    rows(make(), 3)                                          # positions 2 .. 4 of a cache of 4
    with pytest.raises(BackendError, match="position"):
        be.dev_check(0)
    pos.fill_(4)
    be.dev_window_attention_step(make(), P(t), P(t), P(t), None, P(pos), P(out))
    with pytest.raises(BackendError, match="position"):
        be.dev_check(0)


# ---- the decayed write ----
STATES = [
    dict(heads=3, dim=20, vdim=28, decay=[0.9, 0.99, 0.9995], rot=(500.0, 12)), dict(heads=1, dim=32, vdim=32, decay=[1.0], rot=(10.0, 32)), dict(heads=2, dim=130, vdim=65, decay=[0.5, 0.97], rot=(1e4, 130)),
    dict(heads=2, dim=256, vdim=256, decay=[0.999, 1e-3], rot=(1e5, 100)), dict(heads=2, dim=64, vdim=200, decay=[0.98, 0.95], rot=(1e4, 64)),
    dict(heads=4, dim=20, vdim=28, rank=10, tau=8.0), dict(heads=3, dim=64, vdim=33, rank=70, tau=16.0), dict(heads=1, dim=256, vdim=100, rank=300, tau=2.0), dict(heads=2, dim=33, vdim=256, rank=1, tau=1.0),
    dict(heads=2, dim=96, vdim=40, rank=16, tau=1.0, shift=-90.0), dict(heads=5, dim=8, vdim=9, rank=8, tau=16.0, shift=30.0),
]
CUTS = [[75], [2, 3, 40, 7, 9], [1, 8, 16, 17], [33]]


def state_case(be, m):
    """(layer, what keeps its pointers alive, the rows of its projections, a function of projections: the oracle's outputs)"""
    rng, T, eps = np.random.default_rng(m["dim"]), 84, 1e-5
    H, D, V = m["heads"], m["dim"], m["vdim"]
    ranked = "rank" in m
    rows = [("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V)] + ([("a1", m["rank"])] if ranked else [])
    keep = dict(norm=(1 + 0.2 * rng.standard_normal(V)) if ranked else np.ones(V), state=np.zeros((H, V, round_up(D, 32))))
    w, extra, handle, held = {**cases.selectors(rows), "o": np.eye(H * V)}, {}, None, []
    if ranked:
        handle, w["a2"] = bf16_matrix(be, H * D, m["rank"], 7)
        keep["dt_bias"] = rng.standard_normal(H * D) + m.get("shift", 1.0)
        w["a2.b"], w["norm"] = keep["dt_bias"].astype(np.float32), keep["norm"].astype(np.float32)
        extra = dict(a2=handle, inv_tau=1.0 / m["tau"])
        mix = lambda proj: ref.gla(proj, w, dict(heads=H, dim=D, vdim=V, tau=m["tau"]), eps)
    else:
        base, dims = m["rot"]
        held = [dev(t) for t in rotation_tables(Rotation(base, dims), T)]
        keep["decay"] = np.array(m["decay"])
        extra = dict(rot_pairs=dims // 2, max_positions=T, rot_cos=P(held[0]), rot_sin=P(held[1]))
        mix = lambda proj: ref.retention(proj, w, dict(heads=H, dim=D, vdim=V, decay=m["decay"], rot=dict(base=base, dims=dims)), eps)
    d = {n: dev(t) for n, t in keep.items()}
    return LinearLayer(H, H, D, V, 0, eps, **extra, **{n: P(t) for n, t in d.items()}), (d, held), rows, mix, handle


@pytest.mark.parametrize("m", STATES)
def test_decayed_write(be, m):
    layer, (d, _), rows, mix, handle = state_case(be, m)
    H, V, T, N = m["heads"], m["vdim"], 84, sum(n for _, n in rows)
    proj = np.random.default_rng(0).standard_normal((T, N)).astype(np.float32)
    want, dp = mix(proj.astype(np.float64)), dev(proj)
    gate_at = 2 * H * m["dim"] + H * V
    size = be.state_scan_workspace_bytes(layer, DECAYED_WRITE, T)
    ws, o, y, one = zeros(size // 4), zeros(T, H, V), zeros(T, H * V), zeros(H * V)
    for cuts in CUTS:
        d["state"].zero_()
        pos, done, got = dev([0], np.int32), 0, np.zeros_like(want)
        for n in cuts:
            row = P(dp) + 4 * done * N
            be.dev_decayed_write_scan(layer, row, N, n, P(pos), P(ws), size, P(o))
            be.dev_head_outputs_rows(P(o), n, H, V, V, P(y), H * V, False, weight=layer.norm, eps=layer.eps, gate=row + 4 * gate_at, gate_ld=N, gate_mode=3)
            got[done:done + n] = host(y)[:n]
            done += n
            pos.fill_(done)
        while done < T:
            be.dev_state_step(layer, DECAYED_WRITE, P(dp) + 4 * done * N, P(pos), P(one))
            got[done] = host(one)
            done += 1
            pos.fill_(done)
        be.dev_check(0)
        close(got, want, 1e-4)
    with pytest.raises(BackendError):
        be.dev_decayed_write_scan(layer, P(dp), N, T, P(pos), P(ws), size - 4, P(o))
    with pytest.raises(BackendError):
        be.dev_decayed_write_scan(layer, P(dp), N - H * V - m.get("rank", 0) - 1, 1, P(pos), P(ws), size, P(o))
    if handle:
        be.dev_free(handle)


def test_state_keeps_a_write_far_away(be):
    # one token writes, nothing decays and no later key touches its channel: five hundred tokens later the read-out is still exact
    H, D, V, T = 2, 40, 24, 520
    rng = np.random.default_rng(0)
    proj = np.zeros((T, 2 * H * (D + V)), np.float32)
    q, k, v = (proj[:, a:a + H * n].reshape(T, H, n) for a, n in ((0, D), (H * D, D), (2 * H * D, V)))
    k[:, :, 1:], v[:] = rng.standard_normal((T, H, D - 1)), rng.standard_normal((T, H, V))
    k[3], k[3, :, 0] = 0.0, D ** 0.5
    q[:, :, 0] = 1.0
    proj[:, 2 * H * D:2 * H * D + H * V] = v.reshape(T, -1)
    proj[:, :H * D], proj[:, H * D:2 * H * D] = q.reshape(T, -1), k.reshape(T, -1)
    ones, decay, dp, o, pos = dev(np.ones(V)), dev(np.ones(H)), dev(proj), zeros(T, H, V), dev([0], np.int32)
    for cuts in ([T], [5, 515], [4, 2, 2, 512]):
        state = zeros(H, V, 64)
        layer = LinearLayer(H, H, D, V, 0, 1e-5, decay=P(decay), norm=P(ones), state=P(state))
        size, done = be.state_scan_workspace_bytes(layer, DECAYED_WRITE, T), 0
        ws = zeros(size // 4)
        for n in cuts:
            be.dev_decayed_write_scan(layer, P(dp) + 4 * done * proj.shape[1], proj.shape[1], n, P(pos), P(ws), size, P(o) + 4 * done * H * V)
            done += n
        got = host(o)
        assert not got[:3].any()
        close(got[3:], np.broadcast_to(v[3], (T - 3, H, V)), 1e-6)


# ---- whole models ----
def decoder(be, name, dtype="float32", chunk=None, **kw):
    c, cfg, bits, weights = cases.model(name)
    dec = SikivikDecoder(be, cfg, bits.__getitem__, dtype=dtype, **{"max_positions": 640, **kw})
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
    for n in (1, 2):
        dec.reset()
        assert cases.logit_error(dec.feed(ids[:n], list(range(n))), want[:n]) <= bar
    dec.close()


def test_a_sequence_leaves_nothing_behind(be):
    c, weights, dec = decoder(be, "ragged", chunk=64)
    a, b = cases.tokens_for(c, 120, 5), cases.tokens_for(c, 61, 6)
    first = feed_in(dec, b, [40, 1, 20])
    for _ in range(2):
        feed_in(dec, a, [64, 3, 1])                              # a longer sequence fills caches, rings and states
        assert np.array_equal(feed_in(dec, b, [40, 1, 20]), first)
    dec.generate(a[:30], 20)
    assert np.array_equal(feed_in(dec, b, [40, 1, 20]), first)
    assert cases.logit_error(first, ref.forward(c, weights, b)[0]) <= F32_BAR
    dec.close()


def test_unequal_requests_in_turn(be):
    # requests of different lengths one after the other, each as if it were alone
    c, weights, dec = decoder(be, "wide", chunk=32)
    for n, cuts in ((3, [2, 1]), (90, [64, 2]), (1, [1]), (33, [32, 1]), (47, [1])):
        ids = cases.tokens_for(c, n, n)
        assert cases.logit_error(feed_in(dec, ids, cuts), ref.forward(c, weights, ids)[0]) <= F32_BAR, n
    dec.close()


def test_wanted_places(be):
    c, _, dec = decoder(be, "ones", chunk=32)
    ids = cases.tokens_for(c, 70)
    every = feed_in(dec, ids, [70])
    dec.reset()
    assert np.array_equal(dec.feed(ids, [69, 0, 31, 32, 31]), every[[69, 0, 31, 32, 31]])      # any order, block edges, one of them twice
    dec.reset()
    assert dec.feed(ids[:9]).shape == (0, c["vocab"])
    dec.close()


def test_long_decoding(be):
    c, weights, dec = decoder(be, "ragged")
    ids = cases.tokens_for(c, 420, 9)
    want, _ = ref.forward(c, weights, ids)
    assert cases.logit_error(feed_in(dec, ids, [20, 1]), want) <= 2 * F32_BAR
    assert cases.logit_error(feed_in(dec, ids, [420]), want) <= 2 * F32_BAR
    dec.close()


def test_cache_of_just_the_right_size(be):
    c, weights, dec = decoder(be, "wide", max_positions=50)
    ids = cases.tokens_for(c, 50)
    assert cases.logit_error(feed_in(dec, ids, [49, 1]), ref.forward(c, weights, ids)[0]) <= F32_BAR
    with pytest.raises(ValueError):
        dec.feed(ids[:1])
    dec.close()


@pytest.mark.parametrize("name", ["ragged", "ones"])
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
    dec.close()


def test_without_mixed_values(be):
    c, cfg, bits, weights = cases.model("ragged")
    c = json.loads(json.dumps(c))
    c["layers"][4]["mixer"]["v_mix"] = False                     # one mixing layer is left: it mixes with nobody, and its share is not read
    bits = {n: t for n, t in bits.items() if not n.endswith("vmix")}
    dec = SikivikDecoder(be, type(cfg).from_dict(c), bits.__getitem__, dtype="float32", max_positions=64)
    dec.capture()
    ids = cases.tokens_for(c, 50)
    assert cases.logit_error(feed_in(dec, ids, [30, 1, 5, 1]), ref.forward(c, weights, ids)[0]) <= F32_BAR
    dec.close()


def test_missing_and_misshapen_tensors_are_refused(be):
    c, cfg, bits, _ = cases.model("ragged")
    with pytest.raises(KeyError):
        SikivikDecoder(be, cfg, {n: t for n, t in bits.items() if n != "l3.mix.a2.b"}.__getitem__)
    with pytest.raises(ValueError, match="l1.mix.o"):
        SikivikDecoder(be, cfg, {**bits, "l1.mix.o": bits["l1.mix.o"][:-1]}.__getitem__)


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
        read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, c["vocab"])
        assert cases.logit_error(np.concatenate([read(0), read(2), read(3)]), want[[0, 49, 59, 4]]) <= bar
    r = subprocess.run([sys.executable, "-m", "zeninfer_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt-ids", ",".join(map(str, ids)), "--max-new", "6"],
                       cwd=ROOT, text=True, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr
    dec = SikivikDecoder(be, cfg, bits.__getitem__, dtype="float32")
    dec.capture()
    assert [int(t) for t in r.stdout.strip().split(",")] == dec.generate(ids, 6)
    dec.close()
