"""A plain, slow Rimidra in numpy float64: whole sequences, no cache, no batching, one function
per mechanism.  It is the oracle of the Rimidra tests and shares nothing with the package.

Notation: T tokens, rows of every array are tokens.  ``w`` maps checkpoint tensor names to float64
arrays, ``cfg`` is the config.json dictionary, ``p`` a tensor-name prefix, ``m`` a mixer's entry.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def unit_rms(x, eps):
    """Rows (last axis) divided by their root mean square, eps under the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x, weight, eps):
    """The root-mean-square norm whose stored weight is an offset from one."""
    return unit_rms(x, eps) * (1.0 + weight)


# ---------------------------------------------------------------- mixer: attention
def query_temperature(positions, temp):
    """Factor on the query at each position: grows with the logarithm of how many whole runs of
    ``every`` tokens the position has reached."""
    if not temp:
        return np.ones(len(positions))
    return 1.0 + float(temp["coef"]) * np.log(np.floor((positions + 1.0) / float(temp["every"])) + 1.0)


def distance_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def visible_keys(T, window):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < window) if window else True)


def sink_softmax(scores, visible, sink):
    """Softmax over the visible keys of every row with one more term exp(sink) in the denominator."""
    s = np.where(visible, scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.where(visible, np.exp(s - top), 0.0)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def attention(h, w, p, m):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = np.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, d) * query_temperature(pos, m.get("q_temp"))[:, None, None]
    k = (h @ w[p + "k"].T).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    seen = visible_keys(T, int(m["mask"]["size"]) if m.get("mask") else 0)
    away = (pos[:, None] - pos[None, :]).astype(np.float64)
    slopes = distance_slopes(H)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        sc = (q[:, hd] @ k[:, g].T) * float(m["scale"]) - slopes[hd] * away
        out[:, hd] = sink_softmax(sc, seen, float(w[p + "sink"][hd])) @ v[:, g]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---------------------------------------------------------------- mixer: retention
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


def retention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate_halves((h @ w[p + "q"].T).reshape(T, H, d), m.get("rot"))
    k = rotate_halves((h @ w[p + "k"].T).reshape(T, H, d), m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    decay = np.asarray(m["decay"], dtype=np.float64)[:, None, None]
    S, o = np.zeros((H, d, dv)), np.zeros((T, H, dv))
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    o = unit_rms(o, eps).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(scores, top):
    """The ``top`` largest of every row, best first, ties to the lower index."""
    return np.argsort(-scores, axis=-1, kind="stable")[:, :top]


def mixture(h, w, p, f, gaps=None):
    """``gaps`` (a list): gets per token how far the last chosen score is above the best one left out."""
    T, top = h.shape[0], int(f["router"]["top"])
    s = sigmoid(h @ w[p + "router"].T)
    idx = choose(s, top)
    if gaps is not None and top < s.shape[1]:
        best = -np.sort(-s, axis=1)
        gaps.append(best[:, top - 1] - best[:, top])
    out = np.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        t, j = np.nonzero(idx == e)
        if len(t):
            out[t] += expert(h[t] * s[t, e][:, None], w, p + f"e{e}.")
    if f.get("shared"):
        out = out + expert(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ---------------------------------------------------------------- the model
def forward(cfg, w, tokens, return_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence; with ``return_layers`` also the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        src = layer.get("weights_of")
        pre, m, f = f"l{i if src is None else src}.", layer["mixer"], layer.get("mlp")
        h = offset_norm(x, w[pre + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention(h, w, pre + "mix.", m)
        elif layer["type"] == "retention":
            y = retention(h, w, pre + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        if f is not None:
            y = y + (dense(h, w, pre + "mlp.") if f["kind"] == "dense" else mixture(h, w, pre + "mlp.", f, gaps))
        x = x + y
        streams.append(x.copy())
    logits = offset_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(streams)) if return_layers else logits
