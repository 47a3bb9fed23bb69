"""The Tedisun decoder, plain and slow: float64 NumPy over whole sequences, one function per
mechanism, no cache, no batching, nothing shared with the engine.

``cfg`` is the configuration as a dictionary (the keys of config.json), ``W`` maps tensor names
to float64 arrays.  A sequence is a list of token ids; position t is its index.

Notation: T tokens, E the width, R residual streams; per mixer H heads, G key heads, keys of size D,
values of size Dv.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_one_plus(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j); rows before the start are zero."""
    T, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u], axis=0)
    y = np.zeros_like(u)
    for j in range(taps):
        y += padded[j:j + T] * w[:, j]
    return y


# ---- residual streams -----------------------------------------------------------------------

def streams_read(X, w_in):
    """X [T, R, E] -> what a sublayer reads before its norm: sum_r w_in[r] X_r."""
    return np.einsum("r,tre->te", w_in, X)


def streams_write(X, y, w_out, mix):
    """Every stream anew from all old ones and the sublayer's result: X_t = sum_s mix[s, t] X_s + w_out[t] y."""
    return np.einsum("st,nse->nte", mix, X) + w_out[None, :, None] * y[:, None, :]


def gated(y, h, w, b):
    """A sublayer's result times the sigmoid of a projection of what the sublayer read."""
    return y * sigmoid(h @ w.T + b)


# ---- gated delta rule -------------------------------------------------------------------------

def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_scan(q, k, v, beta, g):
    """q, k [T, H, D] (unit length, q already scaled), v [T, H, Dv], beta, g [T, H]; per head
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  Returns [T, H, Dv]."""
    T, H, D = q.shape
    o = np.zeros_like(v)
    for h in range(H):
        S = np.zeros((D, v.shape[2]))
        for t in range(T):
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + np.outer(k[t, h], u)
            o[t, h] = S.T @ q[t, h]
    return o


def delta_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda n: silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"]))
    rep = np.arange(H) // (H // G)
    q = unit(conv(".q").reshape(T, G, D))[:, rep] * D ** -0.5
    k = unit(conv(".k").reshape(T, G, D))[:, rep]
    v = conv(".v").reshape(T, H, Dv)
    beta = sigmoid(h @ W[p + ".b"].T)
    g = np.exp(-np.exp(W[p + ".A_log"]) * softplus(h @ W[p + ".a"].T + W[p + ".dt_bias"]))
    o = rms_unit(delta_scan(q, k, v, beta, g), eps) * W[p + ".norm"]
    return (o * silu(h @ W[p + ".g"].T).reshape(T, H, Dv)).reshape(T, H * Dv) @ W[p + ".o"].T


# ---- attention ---------------------------------------------------------------------------------

def banded_frequencies(base, dims, scaling):
    """base^(-2i / dims) for i < dims / 2.  With ``scaling`` (factor, low, high, original) a frequency whose
    wavelength is under original / high stays, one whose wavelength is over original / low is divided by
    factor, and those between are blended linearly in original / wavelength."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f
    factor, low, high, original = (float(scaling[n]) for n in ("factor", "low", "high", "original"))
    out = []
    for v in f:
        wave = 2.0 * math.pi / v
        if wave < original / high:
            out.append(v)
        elif wave > original / low:
            out.append(v / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * v / factor + s * v)
    return np.array(out)


def rotate_halves(x, rot, positions):
    """Turn the first ``rot.dims`` entries of the last axis of x [T, heads, n]; entry i pairs with i + dims / 2."""
    dims = rot["dims"]
    half = dims // 2
    a = np.asarray(positions, dtype=np.float64)[:, None] * banded_frequencies(rot["base"], dims, rot.get("scaling"))[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def visible(i, j, size, keep_first):
    """Whether position i sees position j: j is not later, and lies in the window or among the first tokens."""
    return (j <= i) & ((size == 0) | (i - j < size) | (j < keep_first))


def sink_window_attention(q, k, v, scale, sink, size, keep_first):
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; softmax over the visible keys with exp(sink_h) once more in
    the denominator.  Returns [T, H, Dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    seen = visible(np.arange(T)[:, None], np.arange(T)[None, :], size, keep_first)
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        m = np.maximum(s.max(axis=1, keepdims=True), sink[h])
        e = np.exp(s - m)
        out[:, h] = (e @ v[:, g]) / (e.sum(axis=1, keepdims=True) + np.exp(sink[h] - m))
    return out


def attention_side(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda n: h @ W[p + n].T + W[p + n + ".b"]
    q = rms_unit(lin(".q").reshape(T, H, D), eps) * W[p + ".q.norm"]
    k = rms_unit(lin(".k").reshape(T, G, D), eps) * W[p + ".k.norm"]
    v = lin(".v").reshape(T, G, Dv)
    q, k = rotate_halves(q, m["rot"], np.arange(T)), rotate_halves(k, m["rot"], np.arange(T))
    mask = m.get("mask") or {}
    o = sink_window_attention(q, k, v, m["scale"], W[p + ".sink"], mask.get("size", 0), mask.get("keep_first", 0))
    return o.reshape(T, H * Dv) @ W[p + ".o"].T + W[p + ".o.b"]


# ---- matrix memory -----------------------------------------------------------------------------

def matrix_memory_scan(q, k, v, i, f):
    """q (scaled), k [T, H, D], v [T, H, Dv], log gates i, f [T, H].  With the running maximum m (0 at the
    start): m' = max(f + m, i); S' = exp(f + m - m') S + exp(i - m') k v^T; n' likewise with k alone;
    o = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6).  Returns [T, H, Dv]."""
    T, H, D = q.shape
    o = np.zeros_like(v)
    for h in range(H):
        S, n, m = np.zeros((D, v.shape[2])), np.zeros(D), 0.0
        for t in range(T):
            m_new = max(f[t, h] + m, i[t, h])
            a, b = math.exp(f[t, h] + m - m_new), math.exp(i[t, h] - m_new)
            S = a * S + b * np.outer(k[t, h], v[t, h])
            n = a * n + b * k[t, h]
            m = m_new
            o[t, h] = S.T @ q[t, h] / (max(abs(n @ q[t, h]), math.exp(-m)) + 1e-6)
    return o


def soft_capped(z, cap):
    return cap * np.tanh(z / cap)


def matrix_memory_side(h, W, p, m, eps):
    T = h.shape[0]
    H, D, Dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W[p + ".q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W[p + ".k"].T).reshape(T, H, D)
    v = (h @ W[p + ".v"].T).reshape(T, H, Dv)
    i = soft_capped(h @ W[p + ".i"].T + W[p + ".i.b"], cap)
    f = log_sigmoid(soft_capped(h @ W[p + ".f"].T + W[p + ".f.b"], cap))
    o = rms_unit(matrix_memory_scan(q, k, v, i, f), eps).reshape(T, H * Dv)
    return (o * W[p + ".norm"] * sigmoid(h @ W[p + ".g"].T)) @ W[p + ".o"].T


def parallel_mixer(h, W, p, m, eps):
    """Both sides read h; their results times the sides' scales, added."""
    return (m["left_scale"] * attention_side(h, W, p + ".left", m["left"], eps)
            + m["right_scale"] * matrix_memory_side(h, W, p + ".right", m["right"], eps))


# ---- mixture of experts ------------------------------------------------------------------------

def route(h, W, p, top):
    """(ids, weights) [T, top]: softmax scores over all rows of the router; the correction moves the choice only."""
    z = h @ W[p + ".router"].T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s /= s.sum(axis=-1, keepdims=True)
    ids = np.argsort(-(s + W[p + ".correction"]), axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def choice_margin(h, W, p, top):
    """How far the last chosen expert's choice score is above the first unchosen one's, per token."""
    z = h @ W[p + ".router"].T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    c = np.sort(s / s.sum(axis=-1, keepdims=True) + W[p + ".correction"], axis=-1)[:, ::-1]
    return c[:, top - 1] - c[:, top] if c.shape[1] > top else np.full(len(c), np.inf)


def experts(h, W, p, m):
    """The chosen experts' outputs, weighted; experts from ``experts`` on return their input."""
    r = m["router"]
    ids, w = route(h, W, p, r["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(ids[t], w[t]):
            if e >= r["experts"]:
                y[t] += we * h[t]
            else:
                q = f"{p}.e{e}"
                y[t] += we * (W[q + ".down"] @ (silu(W[q + ".gate"] @ h[t]) * (W[q + ".up"] @ h[t])))
    return y


# ---- the model ---------------------------------------------------------------------------------

MIXERS = {"delta": delta_mixer, "parallel": parallel_mixer}


def sublayer(X, W, p, n, fn, eps):
    """One sublayer of layer ``p`` around the streams: n is 1 (mixer) or 2 (feed-forward)."""
    hc = f"{p}.hc{n}"
    h = norm_one_plus(streams_read(X, W[hc + ".in"]), W[f"{p}.norm{n}"], eps)
    y = gated(fn(h), h, W[f"{p}.rg{n}"], W[f"{p}.rg{n}.b"])
    return streams_write(X, y, W[hc + ".out"], W[hc + ".mix"]), h


def forward(cfg, W, tokens, trace=None, margins=None):
    """Logits [T, vocab] of a whole sequence.  ``trace``: a list that receives the sum of the streams after
    every layer; ``margins``: a list that receives every router's choice margins."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    X = np.repeat(x[:, None, :], cfg.get("streams", 1), axis=1)
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}"
        X, _ = sublayer(X, W, p, 1, lambda h: MIXERS[spec["type"]](h, W, p + ".mix", spec["mixer"], eps), eps)
        if spec.get("mlp") is not None:
            X, h = sublayer(X, W, p, 2, lambda h: experts(h, W, p + ".mlp", spec["mlp"]), eps)
            if margins is not None:
                margins.append(choice_margin(h, W, p + ".mlp", spec["mlp"]["router"]["top"]))
        if trace is not None:
            trace.append(X.sum(axis=1))
    logits = norm_one_plus(X.sum(axis=1), W["final.norm"], eps) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return soft_capped(logits, cap) if cap else logits
