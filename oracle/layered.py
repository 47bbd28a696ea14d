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


def parallel_layers(cfg, w, tokens, layers_out):
    """The residual stream behind post-normed layers of two branches (Mitotar)."""
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
    return rms_norm(x, w["final.norm"], eps, around_zero=True)


# ---- Kuzipel ---------------------------------------------------------------------------------------

def silu(z):
    return z * sigmoid(z)


def layer_norm(x, w, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def rotate(x, p, base):
    """Rotary positions over the whole last axis, element i with element i + half; p one position per row."""
    half = x.shape[-1] // 2
    a = np.asarray(p, np.float64)[:, None] * base ** (-2.0 * np.arange(half) / (2 * half))
    a = a.reshape(a.shape[0], *[1] * (x.ndim - 2), half)
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], axis=-1)


def softmax(z):
    e = np.exp(z - np.max(z, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def causal_softmax(s):
    n = s.shape[-1]
    return softmax(np.where(np.arange(n)[None] <= np.arange(n)[:, None], s, -np.inf))


def latent_attention(h, w, p, eps):
    """Queries, keys and values through low-rank latents; one rotated key part for all heads."""
    n, H, D, R, C = h.shape[0], p["heads"], p["dim"], p["rot_dim"], p["kv_rank"]
    pos = np.arange(n)
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(n, H, D + R)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :C], w["dkv.norm"], eps)
    kr = rotate(down[:, C:], pos, p["rot"]["base"])
    qr = rotate(q[..., D:], pos, p["rot"]["base"])
    k = (c @ w["uk"].T).reshape(n, H, D)
    v = (c @ w["uv"].T).reshape(n, H, p["vdim"])
    out = np.empty((n, H, p["vdim"]))
    for a in range(H):
        out[:, a] = causal_softmax((q[:, a, :D] @ k[:, a].T + qr[:, a] @ kr.T) * p["scale"]) @ v[:, a]
    return out.reshape(n, -1) @ w["o"].T


def token_shift(h, mu):
    """Each token's vector moved by mu towards the one before it (zeros before the first)."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def channel_decay(z, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(z @ w1.T) @ w2.T + w0))


def wkv_step(S, r, k, v, w, u):
    """One token of one head.  S [key channel, value channel]."""
    kv = np.outer(k, v)
    o = (S + u[:, None] * kv).T @ r
    return w[:, None] * S + kv, o


def wkv(h, w, p, eps):
    n, H, D = h.shape[0], p["heads"], p["dim"]
    mixed = {t: token_shift(h, w["mu." + t]) for t in "rkvgw"}
    r, k, v = ((mixed[t] @ w[t].T).reshape(n, H, D) for t in "rkv")
    d = channel_decay(mixed["w"], w["w1"], w["w2"], w["w0"]).reshape(n, H, D)
    u = w["u"].reshape(H, D)
    out = np.empty((n, H, D))
    for a in range(H):
        S = np.zeros((D, D))
        for t in range(n):
            S, out[t, a] = wkv_step(S, r[t, a], k[t, a], v[t, a], d[t, a], u[a])
    y = unit_rms(out, eps).reshape(n, H * D) * w["norm"] * silu(mixed["g"] @ w["g"].T)
    return y @ w["o"].T


def glu(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z, top):
    """Weights [n, experts]: softmax over the `top` largest logits of each row, zero elsewhere."""
    out = np.zeros_like(z)
    for t in range(z.shape[0]):
        chosen = np.argsort(-z[t], kind="stable")[:top]
        out[t, chosen] = softmax(z[t, chosen])
    return out


def mixture(h, w, p):
    g = route(h @ w["router"].T + w["router.b"], p["router"]["top"])
    y = sum(g[:, [e]] * glu(h, under(w, f"e{e}.")) for e in range(p["router"]["experts"]))
    return y + sigmoid(h @ w["shared.sg"].T) * glu(h, under(w, "shared."))


def layer_runs(n_layers, loop):
    """(layer, does a pass of the loop begin before it) in the order of computation."""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    body = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body * loop["times"] + [(i, False) for i in range(b, n_layers)]


MIXERS = {"latent_attention": latent_attention, "wkv": wkv}


def prenorm_layers(cfg, w, tokens, layers_out):
    """The residual stream behind pre-normed layers with layer scale, some of them in a loop (Kuzipel)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = x = w["embed"][np.asarray(tokens)]
    for i, begins in layer_runs(len(cfg["layers"]), cfg.get("loop")):
        if begins:
            x = np.concatenate([x, x0], axis=-1) @ w["loop.in"].T
        layer, lw = cfg["layers"][i], under(w, f"l{i}.")
        x = x + m * lw["ls1"] * MIXERS[layer["type"]](layer_norm(x, lw["norm1"], eps), under(lw, "mix."), layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + m * lw["ls2"] * mixture(layer_norm(x, lw["norm2"], eps), under(lw, "mlp."), layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.copy())
    return layer_norm(x, w["final.norm"], eps)


DESIGNS = {"Mitotar": parallel_layers, "Kuzipel": prenorm_layers}


def forward(cfg: dict, weights: dict, tokens, layers_out: list | None = None) -> np.ndarray:
    """Logits [n, vocab] of the whole sequence at once."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    return DESIGNS[cfg.get("architecture", "Mitotar")](cfg, w, tokens, layers_out) @ w["head"].T
