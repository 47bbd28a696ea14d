"""Plain CPU implementation of layer-described models (numpy, float64): one function per mechanism,
token by token where the mechanism is a recurrence, whole score matrices where it is attention.

It is the oracle of the layered engine's tests.  It shares nothing with the product: no kernel, no
weight layout, no chunking, no cache.  Weights are a dict name -> array ([out, in] matrices).
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, np.float64)))


def log_sigmoid(z):
    z = np.asarray(z, np.float64)
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps, around_zero=False):
    return unit_rms(x, eps) * ((1.0 + w) if around_zero else w)


def sinusoid(p, width, base=10000.0):
    v = np.empty(width)
    for c in range(width):
        a = p * base ** (-(c - c % 2) / width)
        v[c] = math.cos(a) if c % 2 else math.sin(a)
    return v


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1)


def distance_slopes(n_heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads)])


def gate_weights(q, k, scale, slopes, head_bias):
    """Sigmoid weights [heads, i, j] of normalised queries [n, heads, dim] against normalised keys
    [n, kv, dim]; zero above the diagonal."""
    n, H, _ = q.shape
    kv = k.shape[1]
    out = np.zeros((H, n, n))
    i, j = np.meshgrid(np.arange(n), np.arange(n), indexing="ij")
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // kv)].T) * scale - slopes[h] * (i - j) + head_bias[h]
        out[h] = np.where(j <= i, sigmoid(s), 0.0)
    return out


def talking_attention(h, w, p, eps):
    """Sigmoid attention whose values are the raw keys and whose heads' weights are mixed.  h [n, width];
    w the tensors under the mixer's prefix; p the mixer's sizes."""
    n = h.shape[0]
    H, KV, D = p["heads"], p["kv_heads"], p["dim"]
    q = (h @ w["q"].T).reshape(n, H, D)
    k = (h @ w["k"].T).reshape(n, KV, D)
    qn = rms_norm(q, w["q.norm"], eps)
    kn = rms_norm(k, w["k.norm"], eps)
    t = np.array([query_temperature(i, p["q_temp"]["coef"], p["q_temp"]["every"]) for i in range(n)])
    a = gate_weights(qn * t[:, None, None], kn, p["scale"], distance_slopes(H), w["pb"])
    mixed = np.einsum("hg,gij->hij", w["talk"], a)
    o = np.stack([mixed[g] @ k[:, g // (H // KV)] for g in range(H)], axis=1)
    return o.reshape(n, H * D) @ w["o"].T


def mlstm_step(S, nrm, m, q, k, v, i, f):
    """One token of one head's matrix memory.  S [dim, vdim], nrm [dim], m the running maximum."""
    m1 = max(f + m, i)
    keep, add = math.exp(f + m - m1), math.exp(i - m1)
    S = keep * S + add * np.outer(k, v)
    nrm = keep * nrm + add * k
    o = (S.T @ q) / (max(abs(float(nrm @ q)), math.exp(-m1)) + 1e-6)
    return S, nrm, m1, o


def mlstm(h, w, p, eps):
    n = h.shape[0]
    H, D, V, cap = p["heads"], p["dim"], p["vdim"], p["gate_cap"]
    q = (h @ w["q"].T).reshape(n, H, D) / math.sqrt(D)
    k = (h @ w["k"].T).reshape(n, H, D)
    v = (h @ w["v"].T).reshape(n, H, V)
    ig = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    fg = log_sigmoid(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    out = np.empty((n, H, V))
    for a in range(H):
        S, nrm, m = np.zeros((D, V)), np.zeros(D), 0.0
        for t in range(n):
            S, nrm, m, out[t, a] = mlstm_step(S, nrm, m, q[t, a], k[t, a], v[t, a], ig[t, a], fg[t, a])
    y = unit_rms(out, eps).reshape(n, H * V) * w["norm"] * sigmoid(h @ w["g"].T)
    return y @ w["o"].T


def under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel_mixer(h, w, p, eps):
    a = talking_attention(h, under(w, "left."), p["left"], eps)
    b = mlstm(h, under(w, "right."), p["right"], eps)
    return 0.5 * (rms_norm(a, w["left.out"], eps) + rms_norm(b, w["right.out"], eps))


def feed_forward(h, w):
    return gelu_tanh(h @ w["up"].T) @ w["down"].T


def forward(cfg: dict, weights: dict, tokens, layers_out: list | None = None) -> np.ndarray:
    """Logits [n, vocab] of the whole sequence at once."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, width = cfg["norm"]["eps"], cfg["width"]
    x = w["embed"][np.asarray(tokens)] + np.stack([sinusoid(p, width) for p in range(len(tokens))])
    for i, layer in enumerate(cfg["layers"]):
        lw = under(w, f"l{i}.")
        y = parallel_mixer(x, under(lw, "mix."), layer["mixer"], eps)
        x = x + rms_norm(y, lw["norm1"], eps, around_zero=True)
        if layer.get("mlp"):
            x = x + rms_norm(feed_forward(x, under(lw, "mlp.")), lw["norm2"], eps, around_zero=True)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps, around_zero=True) @ w["head"].T
