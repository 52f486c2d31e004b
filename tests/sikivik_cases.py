"""Small Sikivik models and the pieces the CPU and GPU tests share.  Sizes are chosen to differ wherever a kernel could confuse
them, and to leave every tile, vector word and group ragged; one model has everything equal or one."""
from __future__ import annotations

import numpy as np

from dense_helpers import logit_error, selectors, tokens_for  # noqa: F401
from oracle import sikivik as ref
from zeninfer_b200 import blocks
from zeninfer_b200.sikivik import SikivikConfig, random_tensors


def mlp(ff):
    return ff and dict(kind="dense", ff=ff)


def gla(heads, dim, vdim, tau, ff):
    return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=tau), "mlp": mlp(ff)}


def retention(decay, dim, vdim, rot, base, ff):
    return {"type": "retention", "mixer": dict(heads=len(decay), dim=dim, vdim=vdim, decay=decay, rot=dict(base=base, dims=rot)), "mlp": mlp(ff)}


def attention(heads, kv_heads, dim, vdim, window, conv, rot, base, ff, v_mix=True, scale=None):
    return {"type": "attention", "mlp": mlp(ff),
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=1.3 * dim ** -0.5 if scale is None else scale, mask=dict(size=window), conv=conv,
                          rot=dict(base=base, dims=rot), v_mix=v_mix)}


def config(width, vocab, layers, eps=1e-5):
    return dict(architecture="Sikivik", width=width, vocab=vocab, norm=dict(eps=eps), layers=layers)


CASES = {   # name -> (config, rank of the decays)
    "ragged": (config(90, 203, [attention(6, 3, 40, 24, 17, 4, 22, 5e3, None, v_mix=False), retention([0.9, 0.99, 0.999], 20, 28, 12, 500.0, 123),
                                attention(4, 2, 18, 30, 9, 2, 18, 1e4, 61), gla(2, 33, 18, 8.0, None), attention(2, 2, 34, 30, 40, 1, 8, 300.0, 75)]), 10),
    "wide": (config(256, 300, [gla(2, 160, 130, 4.0, 200), attention(4, 1, 136, 72, 33, 5, 64, 1e5, 320), retention([0.97, 0.9995], 64, 200, 64, 1e4, 64),
                               attention(2, 1, 60, 72, 130, 3, 60, 2e4, None)], eps=1e-6), 72),
    "ones": (config(32, 64, [attention(1, 1, 32, 32, 1, 1, 32, 10.0, None), gla(1, 32, 32, 1.0, 32), retention([1.0], 32, 32, 2, 1.0, None)], eps=1e-3), 1),
}


def model(name: str, seed: int = 0):
    """(config dict, SikivikConfig, bf16 tensors, the same tensors in fp32 for the oracle).  Attention's queries are scaled up, so that
    single keys stand out among the visible ones."""
    c, rank = CASES[name]
    cfg = SikivikConfig.from_dict(c)
    bits = random_tensors(cfg, rank, seed)
    for i, layer in enumerate(c["layers"]):
        if layer["type"] == "attention":
            bits[f"l{i}.mix.q"] = blocks.to_bf16(3.0 * blocks.from_bf16(bits[f"l{i}.mix.q"]))
    return c, cfg, bits, {n: blocks.from_bf16(a) for n, a in bits.items()}


def undo_rotation(x, dims, base):
    """The vectors whose rotation is x."""
    T = x.shape[0]
    return np.stack([ref.rotate_half(x[t:t + 1], dims, base, start=-t)[0] for t in range(T)])


def undo_conv(y, taps):
    """The channels whose convolution is y; the last tap is not small."""
    n, u = taps.shape[1], np.zeros_like(y)
    for t in range(y.shape[0]):
        u[t] = y[t]
        for j in range(n - 1):
            if t - (n - 1) + j >= 0:
                u[t] -= taps[:, j] * u[t - (n - 1) + j]
        u[t] /= taps[:, -1]
    return u


def short_taps(channels: int, n: int, rng) -> np.ndarray:
    """Taps [channels, n] that can be undone: the last is one, the others sum to less."""
    w = rng.uniform(-0.6, 0.6, (channels, n)) / max(n - 1, 1)
    w[:, -1] = 1.0
    return w.astype(np.float32)


def standout_projections(T: int, m: dict, planted: list[int], seed: int):
    """(projection rows q | k | v | g, taps): after convolution and rotation the keys at `planted` match every query so well that,
    wherever one is visible, it decides the output: a window that is one position off cannot hide."""
    rng = np.random.default_rng(seed)
    H, G, D, V, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    probe = rng.standard_normal((G, D))
    probe *= np.sqrt(D) / np.linalg.norm(probe, axis=1, keepdims=True)
    q = np.repeat(probe, H // G, axis=0)[None] + 0.2 * rng.standard_normal((T, H, D))
    k = 0.5 * rng.standard_normal((T, G, D)) - probe[None]
    v = rng.standard_normal((T, G, V))
    for n, j in enumerate(planted):
        k[j] = probe * (1.0 + 0.1 * (len(planted) - n))          # the one that leaves first weighs most
        v[j] += 3.0 + n
    turned = [undo_rotation(x, rot["dims"], rot["base"]).reshape(T, -1) for x in (q, k)] + [v.reshape(T, -1)]
    taps = [short_taps(x.shape[1], m["conv"], rng) for x in turned]
    cols = [undo_conv(x, w.astype(np.float64)) for x, w in zip(turned, taps)] + [rng.standard_normal((T, H * V))]
    return np.concatenate(cols, axis=1).astype(np.float32), taps
