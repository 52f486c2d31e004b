"""What the tests of the bfloat16 decoders share: device arrays, tolerances, and feeding a decoder in portions."""
from __future__ import annotations

import numpy as np

from zeninfer_b200 import blocks


def tokens_for(c: dict, n: int, seed: int = 1) -> list[int]:
    return np.random.default_rng(seed).integers(0, c["vocab"], n).tolist()


def selectors(rows: list[tuple[str, int]]) -> dict[str, np.ndarray]:
    """Matrices that pick a tensor's columns out of a projection row: with them a mixer of the oracle reads the same projections
    a kernel is given."""
    total, at, out = sum(n for _, n in rows), 0, {}
    for name, n in rows:
        out[name] = np.eye(total)[at:at + n]
        at += n
    return out


def logit_error(got, ref) -> float:
    """Largest over the positions of rms(got - ref) / rms(ref), mean over the vocabulary taken off."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    d = (got - ref) - (got - ref).mean(axis=-1, keepdims=True)
    r = ref - ref.mean(axis=-1, keepdims=True)
    return float((np.sqrt((d * d).mean(axis=-1)) / np.sqrt((r * r).mean())).max())


def dev(a, dtype=np.float32):
    import torch
    return torch.from_numpy(np.ascontiguousarray(np.asarray(a, dtype))).cuda()


def zeros(*shape):
    import torch
    return torch.zeros(shape, device="cuda")


def host(t):
    import torch
    torch.cuda.synchronize()
    return t.float().cpu().numpy()


def bf16_matrix(be, rows, cols, seed):
    bits = blocks.to_bf16(np.random.default_rng(seed).standard_normal((rows, cols), dtype=np.float32) * np.float32(cols ** -0.5))
    return be.dev_upload("BF16", bits.view(np.uint8), rows, cols), blocks.from_bf16(bits).astype(np.float64)


def close(got, want, tol=2e-5):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, err


def feed_in(dec, ids, cuts):
    """Logits after every token, fed in portions of the given sizes (the last one repeats)."""
    dec.reset()
    rows, done, i = [], 0, 0
    while done < len(ids):
        n = min(cuts[min(i, len(cuts) - 1)], len(ids) - done)
        rows.append(dec.feed(ids[done:done + n], list(range(n))))
        done, i = done + n, i + 1
    return np.concatenate(rows)
