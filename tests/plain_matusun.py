"""A plain, slow Matusun in numpy float64: whole sequences, no cache, no batching, one function
per mechanism.  It is the oracle of the Matusun tests and shares nothing with the package.

Notation: T tokens, rows of every array are tokens.  ``w`` maps checkpoint tensor names to float64
arrays, ``cfg`` is the config.json dictionary, ``p`` a tensor-name prefix, ``m`` a mixer's entry.
"""
from __future__ import annotations

import numpy as np


def silu(x):
    return x / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def unit_rms(x, eps):
    """Rows (last axis) divided by their root mean square, eps under the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


# ---------------------------------------------------------------- parallel residual streams
def contract(streams, w_in):
    """streams [S, T, W] -> what a sublayer's norm reads: their sum with a weight each."""
    return np.einsum("s,stw->tw", w_in, streams)


def spread(streams, mix, w_out, y):
    """New stream t: the old streams s weighted by mix[s, t], plus w_out[t] times the sublayer's result."""
    return np.einsum("sr,stw->rtw", mix, streams) + w_out[:, None, None] * y[None]


# ---------------------------------------------------------------- mixer: selective scan
def causal_conv(x, taps_w, bias):
    """Per channel over time: y[t, c] = b[c] + sum_j taps_w[c, j] x[t - (taps - 1) + j, c], zeros
    before the start; the last tap is the current token's."""
    T, C = x.shape
    taps = taps_w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C)), x], axis=0)
    y = np.tile(bias, (T, 1))
    for j in range(taps):
        y = y + padded[j:j + T] * taps_w[:, j]
    return y


def selective_scan(x, dt, A, B, C, D):
    """Channels evolve alone: S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n, y_c = S[c] . C + D_c x_c."""
    T, I = x.shape
    S, y = np.zeros_like(A), np.zeros((T, I))
    for t in range(T):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba1(h, w, p, m):
    I, N, R = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    xz = h @ w[p + "in"].T
    x, z = silu(causal_conv(xz[:, :I], w[p + "conv"], w[p + "conv.b"])), xz[:, I:]
    low = x @ w[p + "x"].T
    dt = softplus(low[:, :R] @ w[p + "dt"].T + w[p + "dt.b"])
    y = selective_scan(x, dt, -np.exp(w[p + "A_log"]), low[:, R:R + N], low[:, R + N:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


# ---------------------------------------------------------------- mixer: attention
def rotate_halves(x, rot):
    """x [T, heads, size]: channel i of the first ``dims`` is paired with channel i + dims/2 and the
    pair turns by position * base^(-2i/dims); the channels from ``dims`` on pass."""
    if not rot:
        return x
    dims, half = int(rot["dims"]), int(rot["dims"]) // 2
    ang = np.arange(x.shape[0])[:, None] * float(rot["base"]) ** (-2.0 * np.arange(half) / dims)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def visible_keys(T, window):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < window) if window else True)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    # the whole projection is one row of the norm, not a head of it
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    q, k = rotate_halves(q, m.get("rot")), rotate_halves(k, m.get("rot"))
    seen = visible_keys(T, int(m["mask"]["size"]) if m.get("mask") else 0)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        sc = np.where(seen, (q[:, hd] @ k[:, g].T) * float(m["scale"]), -np.inf)
        out[:, hd] = softmax(sc) @ v[:, g]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def expert(h, w, p):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def route(h, w_router, correction, r, gaps=None):
    """Chosen experts and weights [T, top].  Softmax over all of them; the correction moves the choice and not
    the weights, which are normalised over the chosen and scaled.  ``gaps`` (a list): gets per token how far the
    last chosen one was above the best one left out."""
    s, top = softmax(h @ w_router.T), int(r["top"])
    choice = s + correction
    idx = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    if gaps is not None and top < s.shape[1]:
        best = -np.sort(-choice, axis=1)
        gaps.append((best[:, top - 1] - best[:, top]) / s.max(axis=1))
    wgt = np.take_along_axis(s, idx, axis=1)
    return idx, wgt / (wgt.sum(axis=1, keepdims=True) + 1e-20) * float(r.get("scale", 1.0))


def mixture(h, w, p, f, gaps=None):
    r = f["router"]
    E = int(r["experts"])
    idx, wgt = route(h, w[p + "router"], w[p + "correction"], r, gaps)
    out = np.zeros_like(h)
    for e in range(E + int(r.get("identity", 0))):
        t, j = np.nonzero(idx == e)
        if len(t):
            y = expert(h[t], w, p + f"e{e}.") if e < E else h[t]       # the last ones hand their input on
            out[t] += wgt[t, j][:, None] * y
    if f.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------- the model
def passes(cfg):
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(cfg, w, tokens, return_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence; with ``return_layers`` also the sum of the streams after every layer run."""
    eps, S = float(cfg["norm"]["eps"]), int(cfg["streams"])
    x = np.repeat(w["embed"][np.asarray(tokens)][None], S, axis=0)
    after = []
    for i in passes(cfg):
        pre, layer = f"l{i}.", cfg["layers"][i]
        m, f = layer["mixer"], layer.get("mlp")
        h = unit_rms(contract(x, w[pre + "hc1.in"]), eps) * w[pre + "norm1"]
        if layer["type"] == "attention":
            y = attention(h, w, pre + "mix.", m, eps)
        elif layer["type"] == "mamba1":
            y = mamba1(h, w, pre + "mix.", m)
        else:
            raise ValueError(layer["type"])
        x = spread(x, w[pre + "hc1.mix"], w[pre + "hc1.out"], y)
        if f is not None:
            h = unit_rms(contract(x, w[pre + "hc2.in"]), eps) * w[pre + "norm2"]
            x = spread(x, w[pre + "hc2.mix"], w[pre + "hc2.out"], mixture(h, w, pre + "mlp.", f, gaps))
        after.append(x.sum(axis=0))
    logits = unit_rms(x.sum(axis=0), eps) * w["final.norm"] @ w["embed"].T
    return (logits, np.stack(after)) if return_layers else logits
