"""The Nelosun decoder, plain and slow: float64 NumPy over whole sequences, one function per
mechanism, no cache, no batching, nothing shared with the engine.

``cfg`` is the configuration as a dictionary (the keys of config.json), ``W`` maps tensor names
to arrays (float64; the expert tables integers).  A sequence is a list of token ids; position t is
its index.

Notation: T tokens, E the width, H query heads, G key/value heads, D / Dv the query-key and value
sizes per head, R the latent's rank, Dr the rotated size, C the recurrence's channels.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def causal(T):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return j <= i


def softmax_rows(s, visible):
    """Row-wise softmax over the entries where ``visible`` is true; zeros elsewhere."""
    s = np.where(visible, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def softmax_plus_one(s, visible):
    """exp(s_j) / (1 + sum exp(s)): one more entry of score 0 in the denominator, without a value."""
    s = np.where(visible, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def query_temperature(T, coef, every):
    """The factor on q at positions 0 .. T - 1."""
    return np.array([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)])


def attention(h, W, p, m):
    """Grouped causal attention with biases, a temperature on the queries, a one in the denominator and a gate of
    one number per head."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + ".q"].T + W[p + ".q.b"]).reshape(T, H, D)
    k = (h @ W[p + ".k"].T + W[p + ".k.b"]).reshape(T, G, D)
    v = (h @ W[p + ".v"].T + W[p + ".v.b"]).reshape(T, G, Dv)
    temp = m.get("q_temp")
    if temp is not None:
        q = q * query_temperature(T, temp["coef"], temp["every"])[:, None, None]
    gate = sigmoid(h @ W[p + ".g"].T)                     # [T, H]
    out = np.zeros((T, H, Dv))
    for head in range(H):
        g = head // (H // G)
        w = softmax_plus_one((q[:, head] @ k[:, g].T) * m["scale"], causal(T))
        out[:, head] = (w @ v[:, g]) * gate[:, head:head + 1]
    return out.reshape(T, H * Dv) @ W[p + ".o"].T + W[p + ".o.b"]


def rotate_half(x, base, dims, positions):
    """Rotary positions on the first ``dims`` entries of the last axis of x [T, ..., n]: entry i turns
    with entry i + dims / 2 by positions * base^(-2i / dims)."""
    out = x.copy()
    half = dims // 2
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(half)])
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(a).reshape(shape), np.sin(a).reshape(shape)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def latent_attention(h, W, p, m, eps):
    """Attention whose queries come from one small latent and whose keys and values come from another."""
    T, H, D, Dr, Dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    cq = rms_norm(h @ W[p + ".dq"].T, W[p + ".dq.norm"], eps)
    q = (cq @ W[p + ".uq"].T).reshape(T, H, D + Dr)
    down = h @ W[p + ".dkv"].T
    c = rms_norm(down[:, :R], W[p + ".dkv.norm"], eps)
    k_rot = rotate_half(down[:, R:], base, dims, pos)
    q_rot = rotate_half(q[:, :, D:], base, dims, pos)
    k = (c @ W[p + ".uk"].T).reshape(T, H, D)
    v = (c @ W[p + ".uv"].T).reshape(T, H, Dv)
    out = np.zeros((T, H, Dv))
    for head in range(H):
        s = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        out[:, head] = softmax_rows(s, causal(T)) @ v[:, head]
    return out.reshape(T, H * Dv) @ W[p + ".o"].T


def causal_conv(u, w, b):
    """u [T, C], w [C, taps]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j); rows before the start are zero."""
    T, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u], axis=0)
    y = np.tile(np.asarray(b, dtype=np.float64), (T, 1))
    for j in range(taps):
        y += padded[j:j + T] * w[:, j]
    return y


def block_linear(u, w, b):
    """A square matrix per equal part of the channels: w [B, n, n] ([out, in]), b [B, n], u [T, B n]."""
    T, (B, n, _) = u.shape[0], w.shape
    return (np.einsum("tbi,boi->tbo", u.reshape(T, B, n), w) + b).reshape(T, B * n)


def rglru_scan(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam), from S = 0.  Returns S at every token."""
    log_a = -8.0 * r * softplus(lam)
    a, push = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * u
    out, S = np.zeros_like(u), np.zeros(u.shape[1])
    for t in range(u.shape[0]):
        S = a[t] * S + push[t]
        out[t] = S
    return out


def rglru(h, W, p, m):
    y = gelu_tanh(h @ W[p + ".y"].T + W[p + ".y.b"])
    u = causal_conv(h @ W[p + ".x"].T + W[p + ".x.b"], W[p + ".conv"], W[p + ".conv.b"])
    r = sigmoid(block_linear(u, W[p + ".ra"], W[p + ".ra.b"]))
    i = sigmoid(block_linear(u, W[p + ".ri"], W[p + ".ri.b"]))
    return (rglru_scan(u, r, i, W[p + ".lam"]) * y) @ W[p + ".o"].T


def clamped_expert(h, W, p, limit):
    g = np.minimum(h @ W[p + ".gate"].T, limit)
    u = np.clip(h @ W[p + ".up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + ".down"].T


def table_experts(h, ids, W, p, f):
    """Each token's experts stand in a table under its id; every one of them weighs 1 / top."""
    out = np.zeros_like(h)
    table, top = np.asarray(W[p + ".table"]).astype(np.int64), f["router"]["top"]
    for t, token in enumerate(ids):
        for e in table[token]:
            out[t] += clamped_expert(h[t], W, f"{p}.e{e}", f["expert"]["limit"]) / top
    return out


def layer_runs(cfg):
    """The layers in the order in which they run, as (layer, does a pass of the loop begin here?)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for _ in range(loop["times"]):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def mix(h, W, p, layer, eps):
    if layer["type"] == "attention":
        return attention(h, W, p, layer["mixer"])
    if layer["type"] == "latent_attention":
        return latent_attention(h, W, p, layer["mixer"], eps)
    if layer["type"] == "rglru":
        return rglru(h, W, p, layer["mixer"])
    raise ValueError(layer["type"])


def forward(cfg, W, tokens, layers=None):
    """Logits [T, vocab] of a whole sequence; ``layers``, a list, receives the residual stream after every layer run."""
    eps, ids = cfg["norm"]["eps"], np.asarray(tokens)
    x0 = W["embed"][ids] * cfg["embedding"]["scale"]
    x = x0.copy()
    for i, begins in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        if begins:
            x = np.concatenate([x, x0], axis=1) @ W["loop.in"].T
        h = rms_norm(x, W[p + ".norm1"], eps)
        d = mix(h, W, p + ".mix", layer, eps) * W[p + ".ls1"]
        if layer.get("mlp") is not None:
            d = d + table_experts(h, ids, W, p + ".mlp", layer["mlp"]) * W[p + ".ls2"]
        x = x + d
        if layers is not None:
            layers.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T
