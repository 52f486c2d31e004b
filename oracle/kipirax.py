"""A plain, slow Kipirax in numpy float64: one function per mechanism, token by token where the mechanism is a recurrence.

Used by tests only; shares nothing with the product path.  Weights are a dict name -> array (any float dtype); `cfg` is the
model's config.json as a dict.
"""
from __future__ import annotations

import numpy as np

F = np.float64


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    """x over the last axis, divided by its root mean square (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def grouped_rms_norm(x, w, groups, eps):
    """The vector in `groups` equal parts, each by its own root mean square; then the weight over the whole."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms(parts, eps).reshape(x.shape) * w


def token_shift(x, shift):
    """h[t] = x[t] + (x[t - 1] - x[t]) * shift, x[-1] = 0."""
    before = np.concatenate([np.zeros_like(x[:1]), x[:-1]])
    return x + (before - x) * shift


def causal_conv(x, taps):
    """Per channel: y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c], zeros before the start."""
    n = taps.shape[1]
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H].  Per head S [D, V]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, D = q.shape
    V = v.shape[2]
    out = np.zeros((T, H, V), F)
    for h in range(H):
        S = np.zeros((D, V), F)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + np.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def gated_write(q, f, v):
    """q, f [T, H, D], v [T, H, V].  Per head S <- diag(f) S + (1 - f) v^T; o = S^T q."""
    T, H, D = q.shape
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        S = np.zeros((D, v.shape[2]), F)
        for t in range(T):
            S = f[t, h][:, None] * S + np.outer(1.0 - f[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def window_attention(q, k, v, scale, size, keep_first):
    """q [T, H, D], k [T, G, D], v [T, G, V]: distance bias 2^(-8 (h + 1) / H) * (i - j), positions i - size < j <= i and j < keep_first."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), F)
    j = np.arange(T)
    for h in range(H):
        slope = 2.0 ** (-8.0 * (h + 1) / H)
        kh, vh = k[:, h // (H // G)], v[:, h // (H // G)]
        for i in range(T):
            seen = (j <= i) & ((i - j < size) | (j < keep_first))
            s = kh[seen] @ q[i, h] * scale - slope * (i - j[seen])
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ vh[seen]
    return out


def channel_delta(h, w, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mixed = {n: silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv"}
    q = unit(mixed["q"].reshape(T, G, D)) * D ** -0.5
    k = unit(mixed["k"].reshape(T, G, D))
    of = np.arange(H) // (H // G)
    v = mixed["v"].reshape(T, H, V)
    beta = sigmoid(h @ w["b"].T)
    rate = softplus(h @ w["a1"].T @ w["a2"].T + w["dt_bias"]).reshape(T, H, D)
    g = np.exp(-np.exp(w["A_log"])[None, :, None] * rate)
    o = delta_rule(q[:, of], k[:, of], v, g, beta)
    o = rms(o, eps) * w["norm"]
    o = o.reshape(T, H * V) * sigmoid(h @ w["g1"].T @ w["g2"].T)
    return o @ w["o"].T


def parallel_left(h, w, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w["q"].T).reshape(T, H, D), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).reshape(T, G, D), eps) * w["k.norm"]
    v = (h @ w["v"].T).reshape(T, G, V)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w["o"].T


def parallel_right(h, w, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).reshape(T, H, D)
    v = (h @ w["v"].T).reshape(T, H, V)
    f = w["lower"] + (1.0 - w["lower"]) * sigmoid(h @ w["f"].T + w["f.b"])
    o = rms(gated_write(q, f.reshape(T, H, D), v), eps) * w["norm"]
    return o.reshape(T, H * V) @ w["o"].T


def parallel(h, w, m, eps):
    side = lambda s: {n[len(s) + 1:]: t for n, t in w.items() if n.startswith(s + ".")}
    left, right = parallel_left(h, side("left"), m["left"], eps), parallel_right(h, side("right"), m["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


def feed_forward(x, up, down):
    return np.maximum(x @ up.T, 0.0) ** 2 @ down.T


def forward(cfg, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in float64."""
    w = {n: np.asarray(t, F) for n, t in weights.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens] + w["pos"][:len(tokens)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {n[len(p) + 4:]: t for n, t in w.items() if n.startswith(p + "mix.")}
        h = token_shift(x, w[p + "shift"])
        mixer = {"channel_delta": channel_delta, "parallel": parallel}[layer["type"]]
        x = x + grouped_rms_norm(mixer(h, mix, layer["mixer"], eps), w[p + "norm1"], groups, eps)
        if layer["mlp"] is not None:
            x = x + grouped_rms_norm(feed_forward(x, w[p + "mlp.up"], w[p + "mlp.down"]), w[p + "norm2"], groups, eps)
        after.append(x)
    logits = grouped_rms_norm(x, w["final.norm"], groups, eps) @ w["head"].T
    cap = cfg["logit_softcap"]
    return cap * np.tanh(logits / cap), np.stack(after)
