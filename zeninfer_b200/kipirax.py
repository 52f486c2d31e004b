"""Kipirax: a decoder whose layers mix tokens either by a gated delta rule or by windowed attention beside a gated linear
recurrence.

    x = embed[token] + pos[p]
    layer:  h = x + (x_prev - x) * shift          token shift; x_prev is the previous token's x at this layer
            x = x + norm1(mixer(h));  x = x + norm2(W_down relu(W_up x)^2)
    logits = cap * tanh(head norm(x) / cap)

norm is an RMS norm in equal groups of the vector.  The mixers:

    channel_delta   per head S [dim][vdim]: S <- g * S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q, with q, k, v behind short
                    causal convolutions, one decay per key channel, and a low-rank output gate
    parallel        left: softmax attention over a sliding window with kept first tokens and a per-head distance bias;
                    right: S <- f * S + (1 - f) v^T; o = S^T q; the result is half the sum of both, each RMS-normed

A decode step is five launches per layer: the input projections of a mixer are one matrix (rows stacked at load time) whose
product launch also ends the sublayer before it (norm, residual add, token shift); the mixer runs in one launch per branch; the
output projections, the up projection (with norm, residual add and squared ReLU) and the down projection follow.  A block of
tokens runs the same operators as tensor-core products and row kernels; the recurrences scan the block with their state in
registers.  The residual stream, the states, the scores and every norm are fp32 in both.

dtype "bfloat16": block products take bf16 activations with fp32 accumulation, single tokens fp32 activations.  "float32": every
activation and every multiply-add is fp32 (the weights are bf16 in the file, which fp32 holds exactly).
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np

from . import blocks
from .backend import (DELTA_RULE, DENSE_PLAIN, DENSE_SOFTCAP, DENSE_SQUARED_RELU, GATED_WRITE, Backend, LinearLayer, SublayerEnd, WindowAttention)
from .dense_decoder import DenseDecoder, round_up

CHANNEL_DELTA, PARALLEL = "channel_delta", "parallel"


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class WindowConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int

    @property
    def pitch(self) -> int:
        return round_up(max(self.dim, self.vdim), 32)


@dataclass(frozen=True)
class GatedWriteConfig:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowConfig
    right: GatedWriteConfig


@dataclass(frozen=True)
class LayerConfig:
    mixer: DeltaConfig | ParallelConfig
    ff: int | None            # None: no feed-forward


@dataclass(frozen=True)
class KipiraxConfig:
    width: int
    vocab: int
    max_positions: int
    layers: tuple[LayerConfig, ...]
    eps: float
    groups: int
    logit_softcap: float | None

    @classmethod
    def from_dict(cls, c: dict) -> "KipiraxConfig":
        layers = []
        for i, entry in enumerate(c["layers"]):
            m = entry["mixer"]
            if entry["type"] == CHANNEL_DELTA:
                mixer = DeltaConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
                if mixer.heads % mixer.kv_heads:
                    raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key heads")
            elif entry["type"] == PARALLEL:
                a, r = m["left"], m["right"]
                mixer = ParallelConfig(WindowConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), a["mask"]["size"], a["mask"]["keep_first"]),
                                       GatedWriteConfig(r["heads"], r["dim"], r["vdim"]))
                if mixer.left.heads % mixer.left.kv_heads:
                    raise ValueError(f"layer {i}: {mixer.left.heads} query heads over {mixer.left.kv_heads} key/value heads")
            else:
                raise ValueError(f"layer {i}: mixer {entry['type']!r} is not known")
            mlp = entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not known")
            layers.append(LayerConfig(mixer, None if mlp is None else mlp["ff"]))
        cap = c.get("logit_softcap")
        cfg = cls(c["width"], c["vocab"], c["max_positions"], tuple(layers), float(c["norm"]["eps"]), c["norm"]["groups"], None if cap is None else float(cap))
        if cfg.width % cfg.groups:
            raise ValueError(f"width {cfg.width} is not {cfg.groups} equal groups")
        return cfg


# The rows of a mixer's input projection matrix, in order: (tensor, rows).
def delta_rows(m: DeltaConfig, rank_a: int, rank_g: int) -> list[tuple[str, int]]:
    return [("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim), ("b", m.heads), ("a1", rank_a), ("g1", rank_g)]


def parallel_rows(m: ParallelConfig) -> list[tuple[str, int]]:
    a, r = m.left, m.right
    return [("left.q", a.heads * a.dim), ("left.k", a.kv_heads * a.dim), ("left.v", a.kv_heads * a.vdim), ("left.g", a.heads),
            ("right.q", r.heads * r.dim), ("right.f", r.heads * r.dim), ("right.v", r.heads * r.vdim)]


def tensor_plan(cfg: KipiraxConfig, rank_a: int, rank_g: int) -> list[tuple[str, tuple[int, ...]]]:
    """(name, shape) of every tensor of a model file.  The ranks of the decay's and the gate's projections are the file's own
    (the shapes say them); here they describe a model to be made up."""
    W = cfg.width
    plan: list[tuple[str, tuple[int, ...]]] = [("embed", (cfg.vocab, W)), ("pos", (cfg.max_positions, W))]
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        plan += [(p + "norm1", (W,)), (p + "shift", (W,))]
        if isinstance(m, DeltaConfig):
            plan += [(f"{p}mix.{n}", (rows, W)) for n, rows in delta_rows(m, rank_a, rank_g)]
            plan += [(f"{p}mix.{n}.conv", (rows, m.conv)) for n, rows in delta_rows(m, rank_a, rank_g)[:3]]
            plan += [(p + "mix.A_log", (m.heads,)), (p + "mix.norm", (m.vdim,)), (p + "mix.dt_bias", (m.heads * m.dim,)),
                     (p + "mix.a2", (m.heads * m.dim, rank_a)), (p + "mix.g2", (m.heads * m.vdim, rank_g)), (p + "mix.o", (W, m.heads * m.vdim))]
        else:
            plan += [(f"{p}mix.{n}", (rows, W)) for n, rows in parallel_rows(m)]
            plan += [(p + "mix.left.q.norm", (m.left.dim,)), (p + "mix.left.k.norm", (m.left.dim,)), (p + "mix.left.o", (W, m.left.heads * m.left.vdim)),
                     (p + "mix.right.f.b", (m.right.heads * m.right.dim,)), (p + "mix.right.lower", (m.right.heads * m.right.dim,)),
                     (p + "mix.right.norm", (m.right.vdim,)), (p + "mix.right.o", (W, m.right.heads * m.right.vdim)),
                     (p + "mix.left.out", (W,)), (p + "mix.right.out", (W,))]
        if layer.ff is not None:
            plan += [(p + "norm2", (W,)), (p + "mlp.up", (layer.ff, W)), (p + "mlp.down", (W, layer.ff))]
    return plan + [("final.norm", (W,)), ("head", (cfg.vocab, W))]


class KipiraxDecoder(DenseDecoder):
    Config = KipiraxConfig

    def __init__(self, backend: Backend, cfg: KipiraxConfig, tensor, dtype: str = "bfloat16", max_positions: int | None = None, device=None) -> None:
        self._init_dense(backend, cfg, tensor, dtype, min(max_positions or cfg.max_positions, cfg.max_positions), device)
        fetch, matrix, vector = self._fetch, self._matrix, self._vector
        W, add, f32 = cfg.width, self.sequence.add, dict(dtype=self.torch.float32, device=self.dev)

        self.embed = matrix(("embed", cfg.vocab))
        self.positions = matrix(("pos", cfg.max_positions))
        for i, layer in enumerate(cfg.layers):
            p, m = f"l{i}.", layer.mixer
            # `before`: the previous token's x at this layer
            L = dict(shift=vector(p + "shift", (W,)), norm1=vector(p + "norm1", (W,)), before=add(p + "before", (W,), start_zero=True), ff=layer.ff)
            if isinstance(m, DeltaConfig):
                rank_a, rank_g = (fetch(f"{p}mix.{n}").shape[0] for n in ("a1", "g1"))
                rows = delta_rows(m, rank_a, rank_g)
                L.update(proj=matrix(*[(f"{p}mix.{n}", r) for n, r in rows]), o=[matrix((p + "mix.o", W), columns=m.heads * m.vdim)],
                         a2=matrix((p + "mix.a2", m.heads * m.dim), columns=rank_a), g2=matrix((p + "mix.g2", m.heads * m.vdim), columns=rank_g),
                         rank_a=rank_a, rank_g=rank_g)
                conv = self.torch.cat([vector(f"{p}mix.{n}.conv", (r, m.conv)) for n, r in rows[:3]]).t().contiguous()      # [taps][channels]
                keep = dict(conv=conv, a_log=vector(p + "mix.A_log", (m.heads,)), dt_bias=vector(p + "mix.dt_bias", (m.heads * m.dim,)),
                            norm=vector(p + "mix.norm", (m.vdim,)), ring=add(p + "ring", (m.conv, m.channels)),
                            state=add(p + "state", (m.heads, m.vdim, round_up(m.dim, 32)), start_zero=True))
                L["delta"] = LinearLayer(m.heads, m.kv_heads, m.dim, m.vdim, m.conv, cfg.eps, a2=L["a2"], g2=L["g2"], **{n: t.data_ptr() for n, t in keep.items()})
            else:
                a, r = m.left, m.right
                rows = parallel_rows(m)
                L.update(proj=matrix(*[(f"{p}mix.{n}", k) for n, k in rows]),
                         o=[matrix((p + "mix.left.o", W), columns=a.heads * a.vdim), matrix((p + "mix.right.o", W), columns=r.heads * r.vdim)],
                         out=[vector(p + "mix.left.out", (W,)), vector(p + "mix.right.out", (W,))])
                keep = dict(q_weight=vector(p + "mix.left.q.norm", (a.dim,)), k_weight=vector(p + "mix.left.k.norm", (a.dim,)),
                            k_cache=add(p + "k", (self.max_positions, a.kv_heads, a.pitch)), v_cache=add(p + "v", (self.max_positions, a.kv_heads, a.pitch)))
                L["window"] = WindowAttention(a.heads, a.kv_heads, a.dim, a.vdim, a.pitch, a.window, a.keep_first, 1, self.max_positions, a.scale, cfg.eps,
                                              **{n: t.data_ptr() for n, t in keep.items()})
                write = dict(f_bias=vector(p + "mix.right.f.b", (r.heads * r.dim,)), lower=vector(p + "mix.right.lower", (r.heads * r.dim,)),
                             norm=vector(p + "mix.right.norm", (r.vdim,)),
                             state=add(p + "state", (r.heads, r.vdim, round_up(r.dim, 32)), start_zero=True))
                L["write"] = LinearLayer(r.heads, r.heads, r.dim, r.vdim, 0, cfg.eps, **{n: t.data_ptr() for n, t in write.items()})
                keep.update({"right." + n: t for n, t in write.items()})
            # first column of every tensor's outputs in the projection row
            L["at"], total = {}, 0
            for n, k in rows:
                L["at"][n] = total
                total += k
            L["proj_rows"], L["mixer"], L["tensors"] = total, m, keep
            if layer.ff is not None:
                L.update(norm2=vector(p + "norm2", (W,)), up=matrix((p + "mlp.up", layer.ff)), down=matrix((p + "mlp.down", W), columns=layer.ff))
            self.layers.append(L)
        self.final_norm = vector("final.norm", (W,))
        self.head = matrix(("head", cfg.vocab))
        # one token's vectors
        mixed = max(max(m.heads * m.vdim if isinstance(m, DeltaConfig) else max(m.left.heads * m.left.vdim, m.right.heads * m.right.vdim) for m in
                        (layer.mixer for layer in cfg.layers)), 1)
        self.x = [self.torch.zeros(W, **f32) for _ in range(2)]
        self.y = [self.torch.zeros(W, **f32) for _ in range(2)]
        self.proj = self.torch.zeros(max(L["proj_rows"] for L in self.layers), **f32)
        self.mixed = [self.torch.zeros(mixed, **f32) for _ in range(2)]
        self.hidden = self.torch.zeros(max([L["ff"] or 1 for L in self.layers]), **f32)

    # ---- the end of a sublayer: what the next launch that reads the residual stream still has to do ----
    def _end(self, pending: dict, x_out=None, shift_of: dict | None = None, out_norm=None) -> SublayerEnd:
        P = lambda t: None if t is None else t.data_ptr()
        y = pending.get("y", [])
        out = pending.get("out", [None, None])
        return SublayerEnd(P(pending["x"]), P(x_out) if y else None, P(y[0]) if y else None, P(y[1]) if len(y) > 1 else None, P(out[0]), P(out[1]),
                           P(pending.get("norm")), P(pending.get("keep")), P(shift_of["shift"]) if shift_of else None, P(shift_of["before"]) if shift_of else None,
                           P(out_norm), self.cfg.width, self.cfg.groups, self.cfg.eps)

    @staticmethod
    def _after_mixer(L: dict, x, y: list) -> dict:
        return dict(x=x, y=y, norm=L["norm1"], keep=L["before"], **({"out": L["out"]} if len(y) > 1 else {}))

    # ---- one token ----
    def _enqueue_layers(self) -> None:
        be, cfg, st = self.be, self.cfg, self.stream.cuda_stream
        P = lambda t: t.data_ptr()
        be.dev_embed_rows_bf16(self.embed, self.positions, P(self.token), 1, P(self.pos), P(self.x[0]), st)
        cur = 0
        pending = dict(x=self.x[0])

        def product(handle, out, **fold):
            nonlocal cur, pending
            be.dev_dense_gemv([(handle, None, P(out))], st, pre=self._end(pending, self.x[cur ^ 1], **fold.pop("end", {})), **fold)
            if pending.get("y"):
                cur ^= 1
            pending = dict(x=self.x[cur])

        at = lambda L, n: P(self.proj) + 4 * L["at"][n]
        for L in self.layers:
            product(L["proj"], self.proj, end=dict(shift_of=L))
            if "delta" in L:
                be.dev_state_step(L["delta"], DELTA_RULE, P(self.proj), P(self.pos), P(self.mixed[0]), st)
            else:
                be.dev_window_attention_step(L["window"], at(L, "left.q"), at(L, "left.k"), at(L, "left.v"), at(L, "left.g"), P(self.pos), P(self.mixed[0]), st)
                be.dev_state_step(L["write"], GATED_WRITE, at(L, "right.q"), P(self.pos), P(self.mixed[1]), st)
            y = self.y[:len(L["o"])]
            be.dev_dense_gemv([(h, P(m), P(out)) for h, m, out in zip(L["o"], self.mixed, y)], st)
            pending = self._after_mixer(L, self.x[cur], y)
            if L["ff"] is not None:
                product(L["up"], self.hidden, act=DENSE_SQUARED_RELU)
                be.dev_dense_gemv([(L["down"], P(self.hidden), P(self.y[0]))], st)
                pending = dict(x=self.x[cur], y=self.y[:1], norm=L["norm2"])
        if "keep" in pending:      # no feed-forward in the last layer: its shift state is written whether or not the head runs
            be.dev_sublayer_end_rows(self._end(pending, self.x[cur ^ 1]), 1, None, 0, False, st)
            pending = dict(x=self.x[cur ^ 1])
        self.pending = pending     # the same at every step
        be.dev_advance_position(P(self.pos), 1, st)

    def _logit_act(self) -> dict:
        return dict(act=DENSE_PLAIN) if self.cfg.logit_softcap is None else dict(act=DENSE_SOFTCAP, cap=self.cfg.logit_softcap)

    def _enqueue_head(self) -> None:
        st = self.stream.cuda_stream
        self.be.dev_dense_gemv([(self.head, None, self.logits.data_ptr())], st, pre=self._end(self.pending, out_norm=self.final_norm), **self._logit_act())
        self.be.dev_greedy_pick([(self.logits.data_ptr(), self.vocab, 0, self.vocab)], 1, self.token.data_ptr(), st)

    # ---- a block of tokens ----
    def _prefill_buffers(self) -> dict:
        if self._pf is None:
            torch, cfg, T = self.torch, self.cfg, self.PREFILL_CHUNK
            f32 = dict(dtype=torch.float32, device=self.dev)
            view = dict(dtype=torch.float32 if self.exact else torch.bfloat16, device=self.dev)
            deltas = [L["mixer"] for L in self.layers if "delta" in L]
            pairs = [L["mixer"] for L in self.layers if "window" in L]
            most = lambda values: max([1, *values])
            pitch = lambda n: round_up(n, 32)
            row = lambda n: torch.zeros((T, n), **f32)
            self._pf = dict(
                x=[row(cfg.width), row(cfg.width)], y=[row(cfg.width), row(cfg.width)], proj=row(most(L["proj_rows"] for L in self.layers)),
                h=torch.zeros((T, round_up(cfg.width, 8)), **view),
                hidden=torch.zeros((T, round_up(most(L["ff"] or 1 for L in self.layers), 8)), **view),
                mixed=torch.zeros((T, round_up(most([m.heads * m.vdim for m in deltas] + [max(m.left.heads * m.left.vdim, m.right.heads * m.right.vdim) for m in pairs]), 8)), **view),
                low=torch.zeros((T, round_up(most(max(L["rank_a"], L["rank_g"]) for L in self.layers if "delta" in L), 8)), **view),
                q=row(most([m.kv_heads * pitch(m.dim) for m in deltas] + [m.left.heads * m.left.pitch for m in pairs])),
                k=row(most(m.kv_heads * pitch(m.dim) for m in deltas)),
                g=row(most([m.heads * pitch(m.dim) for m in deltas] + [m.right.heads * pitch(m.right.dim) for m in pairs])),
                v=row(most(m.heads * m.vdim for m in deltas)), beta=row(most(m.heads for m in deltas)),
                decay=row(most(m.heads * m.dim for m in deltas)), gate=row(most(m.heads * m.vdim for m in deltas)),
                o=row(most([m.heads * m.vdim for m in deltas] + [max(m.left.heads * m.left.pitch, m.right.heads * m.right.vdim) for m in pairs])),
                # the right branch of a parallel mixer runs beside the left one
                right_q=row(most(m.right.heads * pitch(m.right.dim) for m in pairs)), right_o=row(most(m.right.heads * m.right.vdim for m in pairs)),
                right_mixed=torch.zeros((T, round_up(most(m.right.heads * m.right.vdim for m in pairs), 8)), **view))
            space = lambda kind, rule: torch.zeros(most(self.be.state_scan_workspace_bytes(L[kind], rule, T) for L in self.layers if kind in L), dtype=torch.uint8, device=self.dev)
            self._pf.update(scan=space("delta", DELTA_RULE), right_scan=space("write", GATED_WRITE))
            self.side = torch.cuda.Stream(device=self.dev)
            self._fork, self._join = torch.cuda.Event(), torch.cuda.Event()
        return self._pf

    def prefill(self, d_tokens, count: int) -> None:
        be, cfg, st, T, b = self.be, self.cfg, self.stream.cuda_stream, count, self._prefill_buffers()
        if not 1 <= T <= self.PREFILL_CHUNK:
            raise ValueError(f"a block of {T} tokens")
        P = lambda t: t.data_ptr()
        bf16, W = not self.exact, cfg.width
        ld = lambda n: round_up(n, 8)

        def gemm(handle, x, x_ld, out, out_ld, to_view=False, **kw):
            be.dev_dense_gemm(handle, x, x_ld, T, out, out_ld, st, out_bf16=bf16 and to_view, exact=self.exact, **kw)

        cur = 0
        be.dev_embed_rows_bf16(self.embed, self.positions, P(d_tokens), T, P(self.pos), P(b["x"][0]), st)
        pending = dict(x=b["x"][0])

        def end(**fold):
            """Ends the sublayer; the next product's input is then in b["h"]."""
            nonlocal cur, pending
            be.dev_sublayer_end_rows(self._end(pending, b["x"][cur ^ 1], **fold), T, P(b["h"]), ld(W), bf16, st)
            if pending.get("y"):
                cur ^= 1
            pending = dict(x=b["x"][cur])

        for L in self.layers:
            m, N = L["mixer"], L["proj_rows"]
            at = lambda n: P(b["proj"]) + 4 * L["at"][n]
            end(shift_of=L)
            gemm(L["proj"], P(b["h"]), ld(W), P(b["proj"]), N)
            if "delta" in L:
                width = m.heads * m.vdim
                for n, rank, handle, out, rows in (("a1", L["rank_a"], L["a2"], b["decay"], m.heads * m.dim), ("g1", L["rank_g"], L["g2"], b["gate"], width)):
                    be.dev_rows_view(at(n), N, rank, T, P(b["low"]), ld(rank), bf16, st)
                    gemm(handle, P(b["low"]), ld(rank), P(out), rows)
                be.dev_delta_inputs_rows(L["delta"], P(b["proj"]), N, P(b["decay"]), m.heads * m.dim, T, P(self.pos), P(b["q"]), P(b["k"]), P(b["g"]), P(b["v"]), P(b["beta"]), st)
                be.dev_state_scan(L["delta"], DELTA_RULE, P(b["q"]), P(b["k"]), P(b["g"]), P(b["v"]), width, P(b["beta"]), T, P(b["scan"]), b["scan"].numel(), P(b["o"]), st)
                be.dev_head_outputs_rows(P(b["o"]), T, m.heads, m.vdim, m.vdim, P(b["mixed"]), ld(width), bf16, st, weight=L["delta"].norm, eps=cfg.eps,
                                         gate=P(b["gate"]), gate_ld=width, gate_mode=2)
                gemm(L["o"][0], P(b["mixed"]), ld(width), P(b["y"][0]), W)
            else:
                a, r = m.left, m.right
                self._fork.record(self.stream)
                self.side.wait_event(self._fork)
                on_side = self.side.cuda_stream
                be.dev_gated_write_inputs_rows(L["write"], at("right.q"), N, T, P(b["right_q"]), P(b["g"]), on_side)
                be.dev_state_scan(L["write"], GATED_WRITE, P(b["right_q"]), None, P(b["g"]), at("right.v"), N, None, T, P(b["right_scan"]), b["right_scan"].numel(), P(b["right_o"]), on_side)
                be.dev_head_outputs_rows(P(b["right_o"]), T, r.heads, r.vdim, r.vdim, P(b["right_mixed"]), ld(r.heads * r.vdim), bf16, on_side, weight=L["write"].norm, eps=cfg.eps)
                self._join.record(self.side)
                be.dev_window_attention_rows(L["window"], at("left.q"), at("left.k"), at("left.v"), N, T, P(self.pos), P(b["q"]), P(b["o"]), st)
                be.dev_head_outputs_rows(P(b["o"]), T, a.heads, a.vdim, a.pitch, P(b["mixed"]), ld(a.heads * a.vdim), bf16, st, gate=at("left.g"), gate_ld=N, gate_mode=1)
                gemm(L["o"][0], P(b["mixed"]), ld(a.heads * a.vdim), P(b["y"][0]), W)
                self.stream.wait_event(self._join)
                gemm(L["o"][1], P(b["right_mixed"]), ld(r.heads * r.vdim), P(b["y"][1]), W)
            pending = self._after_mixer(L, b["x"][cur], b["y"][:len(L["o"])])
            if L["ff"] is not None:
                end()
                gemm(L["up"], P(b["h"]), ld(W), P(b["hidden"]), ld(L["ff"]), to_view=True, act=DENSE_SQUARED_RELU)
                gemm(L["down"], P(b["hidden"]), ld(L["ff"]), P(b["y"][0]), W)
                pending = dict(x=b["x"][cur], y=b["y"][:1], norm=L["norm2"])
        # the block's residual stream after the last layer
        if pending.get("y"):
            be.dev_sublayer_end_rows(self._end(pending, b["x"][cur ^ 1]), T, None, 0, False, st)
            cur ^= 1
        b["last"] = b["x"][cur]
        be.dev_advance_position(P(self.pos), T, st)
        with self.torch.cuda.stream(self.stream):      # what the head reads after a block: the last token's stream, nothing left to add
            self.x[0].copy_(b["last"][T - 1])
        self.pending = dict(x=self.x[0])


def random_tensor(name: str, shape: tuple[int, ...], rng: np.random.Generator) -> np.ndarray:
    """One tensor of a made-up model, fp32: matrices N(0, 1 / columns), norm weights near one, decays, bounds and shifts in their
    usual ranges."""
    z = rng.standard_normal(shape, dtype=np.float32)
    kind = name.split(".", 1)[-1]
    if name in ("embed", "pos"):
        w = z * 0.5
    elif kind == "shift":
        w = 1.0 / (1.0 + np.exp(-z))
    elif kind.endswith("lower"):
        w = 0.9 / (1.0 + np.exp(-z))
    elif kind.endswith("A_log"):
        w = np.log(1.0 + 3.0 * rng.random(shape, dtype=np.float32))
    elif kind.endswith("dt_bias"):
        w = z - 3.0
    elif len(shape) == 2:
        w = z * shape[1] ** -0.5
    else:
        w = z if kind.endswith("f.b") else 1.0 + 0.1 * z
    return w.astype(np.float32)


def random_tensors(cfg: KipiraxConfig, rank_a: int, rank_g: int, seed: int) -> dict[str, np.ndarray]:
    """A made-up model as bfloat16 bit patterns."""
    rng = np.random.default_rng(seed)
    return {name: blocks.to_bf16(random_tensor(name, shape, rng)) for name, shape in tensor_plan(cfg, rank_a, rank_g)}


__all__ = ["KipiraxConfig", "KipiraxDecoder", "random_tensor", "random_tensors", "tensor_plan"]
