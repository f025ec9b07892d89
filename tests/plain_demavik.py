"""A plain, slow Demavik in float64 numpy: one function per mechanism, dense masks, an explicit loop
over tokens for the recurrences and over tokens and experts for the mixture, no cache.  It shares
no code with the engine; the tests hold the engine against it.

``tensors`` maps checkpoint names to float arrays, ``cfg`` is the dict of a config.json.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms_unit(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def causal_conv(x, w, b):
    """x [T, C], w [C, taps]: out_t = b + sum_j w[:, j] * x_(t - taps + 1 + j), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C)), x])
    out = np.zeros_like(x) + b
    for j in range(taps):
        out += padded[j : j + T] * w[:, j]
    return out


# ---------------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The row of the pair table that each token of a sequence takes (Python integers: no overflow)."""
    rows = [buckets]
    for before, now in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * mul_prev + int(now) * mul_cur) % buckets)
    return rows[: len(tokens)]


def embed(cfg, W, tokens):
    e = cfg["embedding"]
    x = W["embed"][np.asarray(tokens)] * e["scale"]
    if e.get("bigram"):
        b = e["bigram"]
        x = x + W["bigram"][np.asarray(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


# ---------------------------------------------------------------------------------- selective scan
def selective_scan(x, dt, A, B, C, D, S=None):
    """x, dt [T, channels], A [channels, N], B, C [T, N]: every channel has N states of its own, decayed
    by exp(dt A).  Returns (outputs [T, channels], last state)."""
    S = np.zeros(A.shape) if S is None else S.copy()
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out, S


def mamba_inputs(h, W, p, m):
    """(x after convolution and silu, z, dt, A, B, C)."""
    inner, N, R = m["inner"], m["state"], m["dt_rank"]
    both = h @ W[p + "in"].T
    x, z = both[:, :inner], both[:, inner:]
    x = silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"]))
    low = x @ W[p + "x"].T
    dt = softplus(low[:, :R] @ W[p + "dt"].T + W[p + "dt.b"])
    return x, z, dt, -np.exp(W[p + "A_log"]), low[:, R : R + N], low[:, R + N :]


def mamba_mixer(h, W, p, m):
    x, z, dt, A, B, C = mamba_inputs(h, W, p, m)
    y, _ = selective_scan(x, dt, A, B, C, W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


# ---------------------------------------------------------------------------------- gated linear attention
def gated_states(q, k, v, alpha, S=None):
    """One head: q, k, alpha [T, D], v [T, V].  The rows of the state decay, k v^T is added, q reads.
    Returns (outputs [T, V], last state [D, V])."""
    S = np.zeros((k.shape[1], v.shape[1])) if S is None else S.copy()
    out = np.zeros((k.shape[0], v.shape[1]))
    for t in range(k.shape[0]):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def gla_decay(h, W, p, m):
    """sigmoid(z)^(1/tau) [T, heads, dim]."""
    z = h @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "a2.b"]
    return np.exp(-softplus(-z) / m["tau"]).reshape(-1, m["heads"], m["dim"])


def gla_mixer(h, W, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, V)
    alpha = gla_decay(h, W, p, m)
    o = np.stack([gated_states(q[:, i], k[:, i], v[:, i], alpha[:, i])[0] for i in range(H)], axis=1)
    o = (rms_unit(o, eps) * W[p + "norm"]).reshape(T, H * V)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---------------------------------------------------------------------------------- attention
def pair_frequencies(rot):
    """Turns per position of the rotated pairs, the slow ones slowed down further."""
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    out = f.copy()
    for i, fi in enumerate(f):
        length = 2.0 * math.pi / fi
        if length < sc["original"] / sc["high"]:
            continue
        if length > sc["original"] / sc["low"]:
            out[i] = fi / sc["factor"]
        else:
            s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
            out[i] = (1.0 - s) * fi / sc["factor"] + s * fi
    return out


def rotate_half(x, rot):
    """x [T, heads, dim]: dim i of the rotated part turns with dim i + dims / 2."""
    f = pair_frequencies(rot)
    half = f.size
    a = np.arange(x.shape[0])[:, None] * f
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half :]], axis=-1)


def attention_keys(h, W, p, m, eps):
    """Normed, rotated keys [T, kv_heads, dim] and values [T, kv_heads, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    k = rms_unit(h @ W[p + "k"].T + W[p + "k.b"], eps) * W[p + "k.norm"]
    v = h @ W[p + "v"].T + W[p + "v.b"]
    return rotate_half(k.reshape(T, G, m["dim"]), m["rot"]), v.reshape(T, G, m["vdim"])


def attend(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, V]: causal softmax attention, heads in groups of H / G."""
    T, H = q.shape[:2]
    group = H // k.shape[1]
    seen = np.tril(np.ones((T, T), bool))
    out = np.zeros((T, H, v.shape[2]))
    for i in range(H):
        s = np.where(seen, q[:, i] @ k[:, i // group].T * scale, -np.inf)
        w = np.exp(s - s.max(axis=-1, keepdims=True))
        out[:, i] = (w / w.sum(axis=-1, keepdims=True)) @ v[:, i // group]
    return out


def attention_mixer(h, W, p, m, eps, keys_values):
    T, H = h.shape[0], m["heads"]
    q = rms_unit(h @ W[p + "q"].T + W[p + "q.b"], eps) * W[p + "q.norm"]
    q = rotate_half(q.reshape(T, H, m["dim"]), m["rot"])
    return attend(q, *keys_values, m["scale"]).reshape(T, H * m["vdim"]) @ W[p + "o"].T


# ---------------------------------------------------------------------------------- experts
def route(h, W, p, r, margins=None):
    """Per token the chosen experts and their weights.  ``margins`` (a list) gets, per token, the gap
    behind the last chosen expert."""
    logits = h @ W[p + "router"].T + W[p + "router.b"]
    picks = []
    for z in logits:
        order = np.argsort(-z, kind="stable")
        chosen = order[: r["top"]]
        if margins is not None:
            margins.append(z[chosen[-1]] - z[order[r["top"]]] if r["top"] < z.size else np.inf)
        w = np.exp(z[chosen] - z[chosen].max())
        picks.append(list(zip(chosen.tolist(), (w / w.sum()).tolist())))
    return picks


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert_mixture(h, W, p, m, margins=None):
    out = np.zeros_like(h)
    for t, pairs in enumerate(route(h, W, p, m["router"], margins)):
        for e, w in pairs:
            out[t] += w * expert(h[t], W, f"{p}e{e}.")
    return out


# ---------------------------------------------------------------------------------- the model
def forward(cfg, W, tokens, collect=None, margins=None):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) gets the stream after every layer, ``margins``
    (a list) per router and token how clear the choice is."""
    eps, step = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(cfg, W, tokens)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "mamba1":
            y = mamba_mixer(x, W, p + "mix.", m)
        elif layer["type"] == "gla":
            y = gla_mixer(x, W, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = attention_keys(x, W, p + "mix.", m, eps)
            y = attention_mixer(x, W, p + "mix.", m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + step * rms_unit(y, eps) * W[p + "norm1"]
        if layer.get("mlp") is not None:
            clear = []
            y = expert_mixture(x, W, p + "mlp.", layer["mlp"], clear)
            if margins is not None:
                margins.append(np.asarray(clear))
            x = x + step * rms_unit(y, eps) * W[p + "norm2"]
        if collect is not None:
            collect.append(x.copy())
    return (rms_unit(x, eps) * W["final.norm"]) @ W["head"].T
