"""Small Kipirax models and the pieces the CPU and GPU tests share.  Sizes are chosen to differ wherever a kernel could confuse
them, and to leave every tile, vector word and chunk ragged."""
from __future__ import annotations

import numpy as np

from dense_helpers import logit_error, selectors, tokens_for  # noqa: F401
from zeninfer_b200 import blocks
from zeninfer_b200.kipirax import KipiraxConfig, random_tensors


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), "mlp": ff and dict(kind="dense", ff=ff)}


def parallel(left, right, ff):
    heads, kv_heads, dim, vdim, scale, size, keep = left
    return {"type": "parallel", "mlp": ff and dict(kind="dense", ff=ff),
            "mixer": {"left": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size, keep_first=keep)),
                      "right": dict(zip(("heads", "dim", "vdim"), right))}}


def config(width, vocab, groups, layers, cap=20.0, eps=1e-5, positions=640):
    return dict(architecture="Kipirax", width=width, vocab=vocab, max_positions=positions, norm=dict(eps=eps, groups=groups), logit_softcap=cap, layers=layers)


CASES = {   # name -> (config, rank of the decays, rank of the output gate)
    "ragged": (config(90, 203, 3, [delta(4, 2, 20, 28, 3, 122), parallel((6, 3, 40, 24, 0.21, 17, 3), (3, 12, 37), None), delta(3, 3, 33, 18, 5, None),
                                   parallel((4, 1, 18, 50, 0.3, 9, 0), (2, 40, 16), 75)]), 10, 7),
    "wide": (config(256, 300, 8, [parallel((2, 1, 136, 72, 0.08, 40, 45), (1, 160, 130), 200), delta(2, 1, 160, 96, 2, 320), delta(1, 1, 64, 200, 4, 64)], cap=7.0), 72, 130),
    "last_bare": (config(64, 97, 1, [delta(8, 8, 16, 16, 1, 96), parallel((8, 2, 32, 32, 0.2, 64, 1), (4, 16, 16), None)], cap=50.0, eps=1e-6), 4, 4),
}


def model(name: str, seed: int = 0):
    """(config dict, KipiraxConfig, bf16 tensors, the same tensors in fp32 for the oracle)"""
    c, rank_a, rank_g = CASES[name]
    cfg = KipiraxConfig.from_dict(c)
    bits = random_tensors(cfg, rank_a, rank_g, seed)
    return c, cfg, bits, {n: blocks.from_bf16(a) for n, a in bits.items()}


def standout_attention(T: int, heads: int, kv_heads: int, dim: int, vdim: int, planted: list[int], seed: int):
    """q, k, v rows in which the keys at `planted` positions match every query so well that, wherever one is visible, it decides
    the output: a mask that is one position off cannot hide.  Norm weights come with it."""
    rng = np.random.default_rng(seed)
    probe = rng.standard_normal((kv_heads, dim))
    q = np.repeat(probe, heads // kv_heads, axis=0)[None] + 0.3 * rng.standard_normal((T, heads, dim))
    k = 0.5 * rng.standard_normal((T, kv_heads, dim)) - probe[None]
    v = rng.standard_normal((T, kv_heads, vdim))
    for n, j in enumerate(planted):
        k[j] = probe * (1.0 + 0.1 * n)
        v[j] += 3.0 + n
    return (q.astype(np.float32), k.astype(np.float32), v.astype(np.float32),
            (1.0 + 0.1 * rng.standard_normal(dim)).astype(np.float32), (1.0 + 0.1 * rng.standard_normal(dim)).astype(np.float32))
