"""Plain, slow oracle of Suselorn: one numpy function per mechanism, float64, no cache, no batch, no
fusion and no code of the product.  A model is a ``config`` dictionary (the layout of config.json) and a
``weights`` dictionary name -> float array.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def tanh_norm(x, alpha, w, b):
    """tanh(alpha x) * w + b: no statistics of x."""
    return np.tanh(alpha * x) * w + b


def rotate_pairs(x, positions, base):
    """x [T, heads, R]: neighbours (2i, 2i + 1) turn by p * base^(-2i/R)."""
    R = x.shape[-1]
    freq = float(base) ** (-2.0 * np.arange(R // 2) / R)
    a = np.asarray(positions, np.float64)[:, None, None] * freq
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * np.cos(a) - x[..., 1::2] * np.sin(a)
    out[..., 1::2] = x[..., 1::2] * np.cos(a) + x[..., 0::2] * np.sin(a)
    return out


def softmax_with_sink(scores, sink):
    """Weights exp(s_j) / (exp(sink) + sum_j exp(s_j)) over the last axis; -inf scores weigh nothing."""
    m = np.maximum(scores.max(-1, keepdims=True), sink)
    e = np.exp(scores - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink - m))


def queries(h, w, p, mix, eps, positions):
    """Two-step query projection -> unrotated [T, H, dim] and rotated [T, H, rot_dim] parts."""
    H, D, R = mix["heads"], mix["dim"], mix["rot_dim"]
    c = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (c @ w[p + "uq"].T).reshape(-1, H, D + R)
    return q[..., :D], rotate_pairs(q[..., D:], positions, mix["rot"]["base"])


def latents(h, w, p, mix, eps, positions):
    """What one token leaves behind: the normalized latent [T, kv_rank] and the shared rotated key part [T, rot_dim]."""
    z = h @ w[p + "dkv"].T
    r = mix["kv_rank"]
    return rms_norm(z[:, :r], w[p + "dkv.norm"], eps), rotate_pairs(z[:, None, r:], positions, mix["rot"]["base"])[:, 0]


def latent_attention(h, w, p, mix, eps):
    """Per head: keys [W_uk c, rotated part], values W_uv c; causal; a sink in the denominator."""
    T, H, D, V = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    at = np.arange(T)
    qn, qr = queries(h, w, p, mix, eps, at)
    c, kr = latents(h, w, p, mix, eps, at)
    k, v = (c @ w[p + "uk"].T).reshape(T, H, D), (c @ w[p + "uv"].T).reshape(T, H, V)
    out = np.zeros((T, H, V))
    for head in range(H):
        s = (qn[:, head] @ k[:, head].T + qr[:, head] @ kr.T) * mix["scale"]
        s = np.where(at[None, :] <= at[:, None], s, -np.inf)
        out[:, head] = softmax_with_sink(s, float(w[p + "sink"][head])) @ v[:, head]
    return out.reshape(T, H * V) @ w[p + "o"].T


def silu_glu(h, w, p):
    g = h @ w[p + "gate"].T + w[p + "gate.b"]
    return (g / (1.0 + np.exp(-g)) * (h @ w[p + "up"].T + w[p + "up.b"])) @ w[p + "down"].T + w[p + "down.b"]


def hyper(streams, w, p, sublayer):
    """streams [S, T, width].  u = sum_s in[s] x_s, y = sublayer(u), x_t <- sum_s mix[s, t] x_s + out[t] y."""
    u = np.einsum("s,std->td", w[p + "in"], streams)
    y = sublayer(u)
    return np.einsum("st,sxd->txd", w[p + "mix"], streams) + w[p + "out"][:, None, None] * y[None]


def layer(streams, w, i, cfg):
    ly, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."

    def norm(u, n):
        return tanh_norm(u, float(np.reshape(w[n + ".alpha"], ())), w[n], w[n + ".b"])
    streams = hyper(streams, w, p + "hc1.",
                    lambda u: w[p + "ls1"] * latent_attention(norm(u, p + "norm1"), w, p + "mix.", ly["mixer"], eps))
    if ly.get("mlp"):
        streams = hyper(streams, w, p + "hc2.", lambda u: w[p + "ls2"] * silu_glu(norm(u, p + "norm2"), w, p + "mlp."))
    return streams


def order(cfg):
    """Layer numbers in the order they run: those of the loop `times` times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, return_layers=False):
    """Logits of every position of one sequence, from its first token on."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    x = w["embed"][np.asarray(tokens)]
    streams = np.stack([x] * cfg["streams"])
    layers = []
    for i in order(cfg):
        streams = layer(streams, w, i, cfg)
        layers.append(streams.sum(0))
    h = tanh_norm(streams.sum(0), float(np.reshape(w["final.norm.alpha"], ())), w["final.norm"], w["final.norm.b"])
    logits = softcap(h @ w["embed"].T, cfg["logit_softcap"])
    return (logits, layers) if return_layers else logits


def greedy(cfg, w, prompt, steps, tie="last"):
    """Greedy continuation by recomputing the whole sequence for every token."""
    seq = list(prompt)
    for _ in range(steps):
        l = forward(cfg, w, seq)[-1]
        best = np.flatnonzero(l == l.max())
        seq.append(int(best[-1] if tie == "last" else best[0]))
    return seq[len(prompt):]
