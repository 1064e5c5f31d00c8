"""Plain, slow oracle of the config-driven decoder: one numpy function per mechanism.

Written from the equations, in float64, without batching, caching or fusion, and without any code of
the product.  A model is a ``config`` dictionary (the layout of config.json) and a ``weights``
dictionary name -> float array.
"""
from __future__ import annotations

import numpy as np


def layer_norm(x, w, eps):
    """y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w over the last axis."""
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    """y = x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_half(x, positions, dims, base):
    """x [T, heads, D]: pair (i, i + dims/2) of the first ``dims`` entries turns by p * base^(-2i/dims)."""
    half = dims // 2
    freq = float(base) ** (-2.0 * np.arange(half) / dims)
    a = np.asarray(positions, np.float64)[:, None, None] * freq
    u, v = x[..., :half], x[..., half:dims]
    out = x.copy()
    out[..., :half] = u * np.cos(a) - v * np.sin(a)
    out[..., half:dims] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(i, j, size, keep_first):
    """Does query position i see key position j?"""
    return j <= i and (i - j < size or j < keep_first)


def attention_core(q, k, v, positions, scale, size, keep_first):
    """q [T, H, D] at ``positions``; k [S, G, D], v [S, G, Dv] at positions 0 .. S-1 -> [T, H, Dv]."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    i, j = np.asarray(positions)[:, None], np.arange(S)[None, :]
    mask = (j <= i) & ((i - j < size) | (j < keep_first))
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = np.where(mask, s, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (e / e.sum(-1, keepdims=True)) @ v[:, g]
    return out


def project_qkv(h, w, p, mix, eps, positions):
    """Queries and keys normalized over the whole projection and rotated; the values are the raw keys."""
    H, G, D = mix["heads"], mix["kv_heads"], mix["dim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = k.reshape(-1, G, D)
    q = rms_norm(q, w[p + "q.norm"], eps).reshape(-1, H, D)
    k = rms_norm(k, w[p + "k.norm"], eps).reshape(-1, G, D)
    rot = mix["rot"]
    return rotate_half(q, positions, rot["dims"], rot["base"]), rotate_half(k, positions, rot["dims"], rot["base"]), v


def attention_mixer(h, w, p, mix, eps):
    T = h.shape[0]
    q, k, v = project_qkv(h, w, p, mix, eps, np.arange(T))
    o = attention_core(q, k, v, np.arange(T), mix["scale"], mix["mask"]["size"], mix["mask"]["keep_first"])
    return o.reshape(T, -1) @ w[p + "o"].T + w[p + "o.b"]


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def silu_expert(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w_router, top):
    """Chosen experts (largest scores first) and their scores, which are the weights as they stand."""
    s = sigmoid(h @ w_router.T)
    order = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return order, np.take_along_axis(s, order, -1)


def moe_ff(h, w, p, mlp):
    out = np.zeros_like(h)
    chosen, weight = route(h, w[p + "router"], mlp["router"]["top"])
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t], weight[t]):
            out[t] += silu_expert((c * h[t])[None], w, f"{p}e{e}.")[0]  # the weight scales the input
    if mlp.get("shared"):
        out += sigmoid(h @ w[p + "shared.sg"].T) * silu_expert(h, w, p + "shared.")
    return out


def layer(x, w, i, cfg):
    ly, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    y = attention_mixer(layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", ly["mixer"], eps)
    mlp = ly.get("mlp")
    if mlp:
        h = layer_norm(x, w[p + "norm2"], eps)
        y = y + (dense_ff(h, w, p + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp))
    return x + y


def forward(cfg, w, tokens, return_layers=False):
    """Logits of every position of one sequence, from its first token on."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    x = w["embed"][np.asarray(tokens)]
    layers = []
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg)
        layers.append(x)
    logits = layer_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T
    return (logits, layers) if return_layers else logits


def greedy(cfg, w, prompt, steps, tie="last"):
    """Greedy continuation by recomputing the whole sequence for every token."""
    seq = list(prompt)
    for _ in range(steps):
        l = forward(cfg, w, seq)[-1]
        best = np.flatnonzero(l == l.max())
        seq.append(int(best[-1] if tie == "last" else best[0]))
    return seq[len(prompt):]
