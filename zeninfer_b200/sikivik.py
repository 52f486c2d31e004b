"""Sikivik: a decoder of parallel layers, the mixer and the feed-forward side by side behind one norm.

    x = embed[token]
    layer:  h = norm1(x);  x = x + mixer(h) + W_down (silu(W_gate h) * W_up h)
    logits = head norm(x)

The mixers:

    gla         per head S [dim][vdim]: S <- diag(a) S + k v^T; o = S^T q, with a decay per key channel,
                a = sigmoid(W_a2 W_a1 h + b)^(1 / tau); o normed per head
    retention   the same with one constant decay per head and q and k rotated by position; o normed per head without a weight
    attention   softmax over a sliding window; q, k and v (with biases) pass a short causal convolution, q and k are rotated; the
                values of every layer that mixes but the first are blended with that first layer's values of the same token

and every mixer's heads are multiplied by a gate of h (silu, or sigmoid for attention) before the output projection.

Since both sublayers read h and their outputs are summed, a layer is two products: one matrix holds the feed-forward's gate and up
rows in pairs and the mixer's projections below them, the other the output projection and, behind it in every row, the down
projection.  A decode step is three launches per layer: the first product (its prologue adds the residual and norms, its epilogue
forms silu(gate) * up), the mixer, the second product.  A block of tokens runs the same two products on the tensor cores, with row
kernels between them; the recurrences scan it with their state in registers.  The residual stream, the states, the decays, the
scores and every norm are fp32.

dtype "bfloat16": block products take bf16 activations with fp32 accumulation, single tokens fp32 activations.  "float32": every
activation and every multiply-add is fp32 (the weights are bf16 in the file, which fp32 holds exactly).
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np

from . import blocks
from .backend import DECAYED_WRITE, Backend, LinearLayer, SublayerEnd, WindowAttention
from .dense_decoder import DenseDecoder, round_up

GLA, RETENTION, ATTENTION = "gla", "retention", "attention"
DEFAULT_POSITIONS = 8192      # the design itself sets no longest sequence


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int


@dataclass(frozen=True)
class StateConfig:
    """gla has tau, retention decay and rot."""
    heads: int
    dim: int
    vdim: int
    tau: float | None = None
    decay: tuple[float, ...] | None = None
    rot: Rotation | None = None

    @property
    def out(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot: Rotation
    conv: int
    v_mix: bool

    @property
    def out(self) -> int:
        return self.heads * self.vdim

    @property
    def pitch(self) -> int:
        return round_up(max(self.dim, self.vdim), 32)


@dataclass(frozen=True)
class LayerConfig:
    mixer: StateConfig | AttentionConfig
    ff: int | None            # None: no feed-forward


@dataclass(frozen=True)
class SikivikConfig:
    width: int
    vocab: int
    layers: tuple[LayerConfig, ...]
    eps: float

    @classmethod
    def from_dict(cls, c: dict) -> "SikivikConfig":
        layers, shared = [], None
        for i, entry in enumerate(c["layers"]):
            m, kind = entry["mixer"], entry["type"]
            rot = None
            if kind != GLA and kind in (RETENTION, ATTENTION):
                rot = Rotation(float(m["rot"]["base"]), int(m["rot"]["dims"]))
                if rot.dims % 2 or not 0 <= rot.dims <= m["dim"]:
                    raise ValueError(f"layer {i}: {rot.dims} rotated dimensions of {m['dim']}")
            if kind == GLA:
                mixer = StateConfig(m["heads"], m["dim"], m["vdim"], tau=float(m["tau"]))
            elif kind == RETENTION:
                mixer = StateConfig(m["heads"], m["dim"], m["vdim"], decay=tuple(float(d) for d in m["decay"]), rot=rot)
                if len(mixer.decay) != mixer.heads:
                    raise ValueError(f"layer {i}: {len(mixer.decay)} decays for {mixer.heads} heads")
            elif kind == ATTENTION:
                mixer = AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), m["mask"]["size"], rot, m["conv"], bool(m.get("v_mix", False)))
                if mixer.heads % mixer.kv_heads:
                    raise ValueError(f"layer {i}: {mixer.heads} query heads over {mixer.kv_heads} key/value heads")
                if mixer.v_mix:
                    if shared not in (None, (mixer.kv_heads, mixer.vdim)):
                        raise ValueError(f"layer {i}: values of {mixer.kv_heads} x {mixer.vdim} cannot be mixed with {shared[0]} x {shared[1]}")
                    shared = (mixer.kv_heads, mixer.vdim)
            else:
                raise ValueError(f"layer {i}: mixer {kind!r} is not known")
            mlp = entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not known")
            layers.append(LayerConfig(mixer, None if mlp is None else mlp["ff"]))
        return cls(c["width"], c["vocab"], tuple(layers), float(c["norm"]["eps"]))

    def first_values(self) -> int | None:
        """The layer whose values later layers mix in."""
        mixing = [i for i, layer in enumerate(self.layers) if isinstance(layer.mixer, AttentionConfig) and layer.mixer.v_mix]
        return mixing[0] if mixing else None


# The rows of a mixer's projections, in order: (tensor, rows).
def projection_rows(m: StateConfig | AttentionConfig, rank: int) -> list[tuple[str, int]]:
    if isinstance(m, AttentionConfig):
        return [("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim), ("g", m.out)]
    rows = [("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.out), ("g", m.out)]
    return rows if m.decay is not None else rows + [("a1", rank)]


def tensor_plan(cfg: SikivikConfig, rank: int) -> list[tuple[str, tuple[int, ...]]]:
    """(name, shape) of every tensor of a model file.  The rank of the decays' projections is the file's own (the shapes say it); here
    it describes a model to be made up."""
    W = cfg.width
    plan: list[tuple[str, tuple[int, ...]]] = [("embed", (cfg.vocab, W))]
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        rows = projection_rows(m, rank)
        plan += [(p + "norm1", (W,))] + [(f"{p}mix.{n}", (r, W)) for n, r in rows] + [(p + "mix.o", (W, m.out))]
        if isinstance(m, AttentionConfig):
            plan += [(f"{p}mix.{n}.b", (r,)) for n, r in rows[:3]] + [(f"{p}mix.{n}.conv", (r, m.conv)) for n, r in rows[:3]] + [(p + "mix.o.b", (W,))]
            if m.v_mix:
                plan += [(p + "mix.vmix", ())]
        elif m.decay is None:
            plan += [(p + "mix.norm", (m.vdim,)), (p + "mix.a2", (m.heads * m.dim, rank)), (p + "mix.a2.b", (m.heads * m.dim,))]
        if layer.ff is not None:
            plan += [(p + "mlp.gate", (layer.ff, W)), (p + "mlp.up", (layer.ff, W)), (p + "mlp.down", (W, layer.ff))]
    return plan + [("final.norm", (W,)), ("head", (cfg.vocab, W))]


def rotation_tables(rot: Rotation, positions: int) -> tuple[np.ndarray, np.ndarray]:
    """cos and sin [positions][dims / 2] of p * base^(-2 i / dims), rounded to fp32 at the end."""
    i = np.arange(rot.dims // 2, dtype=np.float64)
    angle = np.arange(positions, dtype=np.float64)[:, None] * np.power(rot.base, -2.0 * i / max(rot.dims, 1))
    return np.cos(angle).astype(np.float32), np.sin(angle).astype(np.float32)


class SikivikDecoder(DenseDecoder):
    Config = SikivikConfig

    def __init__(self, backend: Backend, cfg: SikivikConfig, tensor, dtype: str = "bfloat16", max_positions: int | None = None, device=None) -> None:
        self._init_dense(backend, cfg, tensor, dtype, max_positions or DEFAULT_POSITIONS, device)
        torch, W, add, f32 = self.torch, cfg.width, self.sequence.add, dict(dtype=self.torch.float32, device=self.dev)
        vector = self._vector
        tables: dict[Rotation, tuple] = {}

        def rotation(rot: Rotation | None) -> tuple:
            """(pairs, cos, sin), one pair of tables for all layers that rotate alike."""
            if rot is None or rot.dims == 0:
                return 0, None, None
            if rot not in tables:
                tables[rot] = tuple(torch.from_numpy(t).to(self.dev) for t in rotation_tables(rot, self.max_positions))
            return rot.dims // 2, *(t.data_ptr() for t in tables[rot])

        self.tables = tables
        self.embed = self._matrix(("embed", cfg.vocab))
        first = cfg.first_values()
        # a token's values of the first mixing layer
        self.values = None if first is None else torch.zeros(cfg.layers[first].mixer.kv_heads * cfg.layers[first].mixer.vdim, **f32)
        for i, layer in enumerate(cfg.layers):
            p, m, ff = f"l{i}.", layer.mixer, layer.ff or 0
            attends = isinstance(m, AttentionConfig)
            rank = self._fetch(p + "mix.a1").shape[0] if not attends and m.decay is None else 0
            rows = projection_rows(m, rank)
            L = dict(mixer=m, ff=ff, norm1=vector(p + "norm1", (W,)), proj_rows=sum(r for _, r in rows), mixed=round_up(m.out, 8) if ff else m.out, at={}, bias=None, o_bias=None)
            col = 0
            for n, r in rows:
                L["at"][n] = col
                col += r
            # gate and up rows in pairs, then the projections; the output projection's columns, then (16-byte aligned) the down projection's
            into = [self._bits(f"{p}mix.{n}", (r, W)) for n, r in rows]
            out = [self._bits(p + "mix.o", (W, m.out))]
            if ff:
                into.insert(0, np.stack([self._bits(p + "mlp.gate", (ff, W)), self._bits(p + "mlp.up", (ff, W))], axis=1).reshape(2 * ff, W))
                out += [np.zeros((W, L["mixed"] - m.out), np.uint16), self._bits(p + "mlp.down", (W, ff))]
            L["into"], L["out"] = self._upload(np.concatenate(into)), self._upload(np.concatenate(out, axis=1))
            L["inner"] = torch.zeros(L["mixed"] + ff, **f32)       # one token's input of the second product
            pairs, cos, sin = rotation(None if not attends and m.rot is None else m.rot)
            if attends:
                channels = L["at"]["g"]
                keep = dict(conv=torch.cat([vector(f"{p}mix.{n}.conv", (r, m.conv)) for n, r in rows[:3]]).t().contiguous(),      # [taps][channels]
                            ring=add(p + "ring", (m.conv, channels)), k_cache=add(p + "k", (self.max_positions, m.kv_heads, m.pitch)),
                            v_cache=add(p + "v", (self.max_positions, m.kv_heads, m.pitch)))
                L["bias"] = torch.cat([vector(f"{p}mix.{n}.b", (r,)) for n, r in rows[:3]] + [torch.zeros(m.out, **f32)])
                L["o_bias"] = vector(p + "mix.o.b", (W,))
                L["values"] = None if not m.v_mix else "keep" if i == first else "mix"
                L["share"] = float(self._values(p + "mix.vmix", ())) if L["values"] == "mix" else 0.0
                L["window"] = WindowAttention(m.heads, m.kv_heads, m.dim, m.vdim, m.pitch, m.window, 0, 0, self.max_positions, m.scale, cfg.eps, rot_pairs=pairs, rot_cos=cos,
                                              rot_sin=sin, taps=m.conv, gate_values=1, v_share=L["share"], **{n: t.data_ptr() for n, t in keep.items()})
                self._point_values(L["window"], L, self.values)
            else:
                keep = dict(norm=vector(p + "mix.norm", (m.vdim,)) if m.decay is None else torch.ones(m.vdim, **f32),
                            state=add(p + "state", (m.heads, m.vdim, round_up(m.dim, 32)), start_zero=True))
                extra = dict(rot_pairs=pairs, rot_cos=cos, rot_sin=sin, max_positions=self.max_positions)
                if m.decay is None:
                    keep["dt_bias"] = vector(p + "mix.a2.b", (m.heads * m.dim,))
                    extra.update(a2=self._matrix((p + "mix.a2", m.heads * m.dim), columns=rank), inv_tau=1.0 / m.tau)
                else:
                    keep["decay"] = torch.tensor(m.decay, **f32)
                L["state"] = LinearLayer(m.heads, m.heads, m.dim, m.vdim, 0, cfg.eps, **extra, **{n: t.data_ptr() for n, t in keep.items()})
            L["tensors"] = keep
            self.layers.append(L)
        self.final_norm = vector("final.norm", (W,))
        self.head = self._matrix(("head", cfg.vocab))
        # one token's vectors
        self.x = [torch.zeros(W, **f32) for _ in range(2)]
        self.y = torch.zeros(W, **f32)
        self.proj = torch.zeros(max(L["proj_rows"] for L in self.layers), **f32)

    @staticmethod
    def _point_values(window: WindowAttention, L: dict, values) -> None:
        window.v_first = values.data_ptr() if L["values"] == "mix" else None
        window.v_keep = values.data_ptr() if L["values"] == "keep" else None

    def _end(self, pending: dict, x_out=None, out_norm=None) -> SublayerEnd:
        """What the next reader of the residual stream still has to do: add the last layer's output, and norm."""
        P = lambda t: None if t is None else t.data_ptr()
        y = pending.get("y")
        return SublayerEnd(x_in=P(pending["x"]), x_out=P(x_out) if y is not None else None, y_a=P(y), out_norm=P(out_norm), n=self.cfg.width, groups=1, eps=self.cfg.eps)

    # ---- one token ----
    def _enqueue_layers(self) -> None:
        be, st = self.be, self.stream.cuda_stream
        P = lambda t: None if t is None else t.data_ptr()
        be.dev_embed_rows_bf16(self.embed, None, P(self.token), 1, None, P(self.x[0]), st)
        cur, pending = 0, dict(x=self.x[0])
        for L in self.layers:
            at = lambda n: P(self.proj) + 4 * L["at"][n]
            be.dev_dense_gemv([(L["into"], None, P(self.proj))], st, pre=self._end(pending, self.x[cur ^ 1], L["norm1"]), bias=P(L["bias"]), gated=P(L["inner"]) + 4 * L["mixed"],
                              gated_pairs=L["ff"])
            cur ^= "y" in pending
            if "window" in L:
                be.dev_window_attention_step(L["window"], at("q"), at("k"), at("v"), at("g"), P(self.pos), P(L["inner"]), st)
            else:
                be.dev_state_step(L["state"], DECAYED_WRITE, P(self.proj), P(self.pos), P(L["inner"]), st)
            be.dev_dense_gemv([(L["out"], P(L["inner"]), P(self.y))], st, bias=P(L["o_bias"]))
            pending = dict(x=self.x[cur], y=self.y)
        self.pending = pending     # the same at every step
        be.dev_advance_position(P(self.pos), 1, st)

    def _enqueue_head(self) -> None:
        st = self.stream.cuda_stream
        self.be.dev_dense_gemv([(self.head, None, self.logits.data_ptr())], st, pre=self._end(self.pending, out_norm=self.final_norm))
        self.be.dev_greedy_pick([(self.logits.data_ptr(), self.vocab, 0, self.vocab)], 1, self.token.data_ptr(), st)

    # ---- a block of tokens ----
    def _prefill_buffers(self) -> dict:
        if self._pf is None:
            torch, cfg, T = self.torch, self.cfg, self.PREFILL_CHUNK
            f32 = dict(dtype=torch.float32, device=self.dev)
            view = dict(dtype=torch.float32 if self.exact else torch.bfloat16, device=self.dev)
            row = lambda n: torch.zeros((T, n), **f32)
            most = lambda values: max([1, *values])
            windows = [L["mixer"] for L in self.layers if "window" in L]
            states = [L for L in self.layers if "state" in L]
            self._pf = dict(x=[row(cfg.width), row(cfg.width)], y=row(cfg.width), proj=row(max(L["proj_rows"] for L in self.layers)),
                            h=torch.zeros((T, round_up(cfg.width, 8)), **view), inner=torch.zeros((T, max(round_up(L["mixed"] + L["ff"], 8) for L in self.layers)), **view),
                            q=row(most(m.heads * m.pitch for m in windows)), o=row(most([m.heads * m.pitch for m in windows] + [L["mixer"].out for L in states])),
                            values=None if self.values is None else row(self.values.numel()),
                            scan=torch.zeros(most(self.be.state_scan_workspace_bytes(L["state"], DECAYED_WRITE, T) for L in states), dtype=torch.uint8, device=self.dev))
            for L in self.layers:
                if "window" in L:      # the same layer, with a block's values
                    L["window_rows"] = WindowAttention.from_buffer_copy(L["window"])
                    self._point_values(L["window_rows"], L, self._pf["values"])
        return self._pf

    def prefill(self, d_tokens, count: int) -> None:
        be, cfg, st, T, b = self.be, self.cfg, self.stream.cuda_stream, count, self._prefill_buffers()
        if not 1 <= T <= self.PREFILL_CHUNK:
            raise ValueError(f"a block of {T} tokens")
        P = lambda t: None if t is None else t.data_ptr()
        bf16, W = not self.exact, cfg.width
        item = 2 if bf16 else 4
        cur = 0
        be.dev_embed_rows_bf16(self.embed, None, P(d_tokens), T, None, P(b["x"][0]), st)
        pending = dict(x=b["x"][0])
        for L in self.layers:
            m, N, ld = L["mixer"], L["proj_rows"], round_up(L["mixed"] + L["ff"], 8)
            at = lambda n: P(b["proj"]) + 4 * L["at"][n]
            be.dev_sublayer_end_rows(self._end(pending, b["x"][cur ^ 1], L["norm1"]), T, P(b["h"]), round_up(W, 8), bf16, st)
            cur ^= "y" in pending
            be.dev_dense_gemm(L["into"], P(b["h"]), round_up(W, 8), T, P(b["proj"]), N, st, exact=self.exact, bias=P(L["bias"]), gated=P(b["inner"]) + item * L["mixed"],
                              gated_ld=ld, gated_pairs=L["ff"])
            if "window" in L:
                be.dev_window_attention_rows(L["window_rows"], at("q"), at("k"), at("v"), N, T, P(self.pos), P(b["q"]), P(b["o"]), st)
                heads = dict(head_ld=m.pitch, gate_mode=2)
            else:
                be.dev_decayed_write_scan(L["state"], P(b["proj"]), N, T, P(self.pos), P(b["scan"]), b["scan"].numel(), P(b["o"]), st)
                heads = dict(head_ld=m.vdim, gate_mode=3, weight=L["state"].norm, eps=cfg.eps)
            be.dev_head_outputs_rows(P(b["o"]), T, m.heads, m.vdim, heads.pop("head_ld"), P(b["inner"]), ld, bf16, st, gate=at("g"), gate_ld=N, fill=L["mixed"], **heads)
            be.dev_dense_gemm(L["out"], P(b["inner"]), ld, T, P(b["y"]), W, st, exact=self.exact, bias=P(L["o_bias"]))
            pending = dict(x=b["x"][cur], y=b["y"])
        # the block's residual stream after the last layer
        be.dev_sublayer_end_rows(self._end(pending, b["x"][cur ^ 1]), T, None, 0, False, st)
        b["last"] = b["x"][cur ^ 1]
        be.dev_advance_position(P(self.pos), T, st)
        with self.torch.cuda.stream(self.stream):      # what the head reads after a block: the last token's stream, nothing left to add
            self.x[0].copy_(b["last"][T - 1])
        self.pending = dict(x=self.x[0])


def random_tensor(name: str, shape: tuple[int, ...], rng: np.random.Generator) -> np.ndarray:
    """One tensor of a made-up model, fp32: matrices N(0, 1 / columns), norm weights near one, small biases, decays in their usual
    range."""
    z = rng.standard_normal(shape, dtype=np.float32)
    kind = name.split(".", 1)[-1]
    if name == "embed":
        w = z * 0.5
    elif kind.endswith("vmix"):
        w = 0.3 + 0.4 * rng.random(shape, dtype=np.float32)
    elif kind.endswith("a2.b"):
        w = z + 1.0
    elif kind.endswith(".b"):
        w = 0.2 * z
    elif len(shape) == 2:
        w = z * shape[1] ** -0.5
    else:
        w = 1.0 + 0.1 * z
    return np.asarray(w, np.float32)


def random_tensors(cfg: SikivikConfig, rank: int, seed: int) -> dict[str, np.ndarray]:
    """A made-up model as bfloat16 bit patterns."""
    rng = np.random.default_rng(seed)
    return {name: blocks.to_bf16(random_tensor(name, shape, rng)) for name, shape in tensor_plan(cfg, rank)}


__all__ = ["SikivikConfig", "SikivikDecoder", "random_tensor", "random_tensors", "rotation_tables", "tensor_plan"]
