"""Small random models described layer by layer, as folders a loader reads, for the parity tests."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

from oracle import layered as L


def bf16(a) -> np.ndarray:
    """fp32 values rounded to what bf16 can hold (nearest even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def layer(heads, kv_heads, dim, scale, coef, every, mem_heads, mem_dim, mem_vdim, cap, ff):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                               "q_temp": {"coef": coef, "every": every}},
                      "right": {"heads": mem_heads, "dim": mem_dim, "vdim": mem_vdim, "gate_cap": cap}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, eps, layers):
    return {"architecture": "Mitotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


# Sizes that no tile divides, unequal layers, a layer without feed-forward, one head, more heads than the
# tensor-core attention takes.
CONFIGS = {
    "mixed": config(80, 97, 1e-5, [layer(6, 3, 20, 0.3, 0.9, 7, 3, 24, 40, 5.0, 112),
                                   layer(4, 1, 32, 0.2, 0.3, 50, 1, 72, 16, 9.0, 0)]),
    "one_head": config(136, 61, 1e-6, [layer(1, 1, 16, 0.25, 0.0, 1, 1, 8, 96, 3.0, 40)]),
    "many_heads": config(72, 70, 1e-3, [layer(20, 20, 12, 0.5, 0.4, 33, 2, 130, 70, 12.0, 65),
                                        layer(16, 4, 72, 0.1, 0.2, 5, 5, 16, 16, 12.0, 200)]),
    "beyond_tc": config(96, 83, 1e-5, [layer(40, 8, 8, 0.4, 0.5, 20, 2, 64, 64, 8.0, 96)]),
    "odd": config(75, 53, 1e-5, [layer(3, 1, 15, 0.3, 0.7, 11, 3, 9, 33, 4.0, 101), layer(5, 5, 7, 0.6, 0.2, 3, 1, 65, 5, 4.0, 0)]),
    "wide_keys": config(64, 40, 1e-5, [layer(16, 16, 256, 0.06, 0.4, 17, 1, 12, 12, 6.0, 32)]),
    "pairs": config(64, 50, 1e-5, [layer(2, 2, 136, 0.08, 0.5, 9, 2, 40, 24, 6.0, 48)]),
}


def weights(cfg, seed=0):
    """name -> fp32 array holding bf16 values."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    w = {}

    def mat(name, r, c, s=1.0):
        w[name] = bf16(s * rng.standard_normal((r, c)) / np.sqrt(c))

    def vec(name, n, mean, s=0.3):
        w[name] = bf16(mean + s * rng.standard_normal(n))

    w["embed"] = bf16(1.5 * rng.standard_normal((cfg["vocab"], W)))
    for i, l in enumerate(cfg["layers"]):
        p, a, m = f"l{i}.", l["mixer"]["left"], l["mixer"]["right"]
        vec(p + "norm1", W, 0.0)
        mat(p + "mix.left.q", a["heads"] * a["dim"], W)
        mat(p + "mix.left.k", a["kv_heads"] * a["dim"], W)
        vec(p + "mix.left.q.norm", a["dim"], 1.0)
        vec(p + "mix.left.k.norm", a["dim"], 1.0)
        w[p + "mix.left.talk"] = bf16(np.eye(a["heads"]) + 0.4 * rng.standard_normal((a["heads"],) * 2))
        vec(p + "mix.left.pb", a["heads"], -1.0, 1.0)
        mat(p + "mix.left.o", W, a["heads"] * a["dim"])
        vec(p + "mix.left.out", W, 1.0)
        for t, n in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
            mat(p + "mix.right." + t, m["heads"] * n, W)
        mat(p + "mix.right.o", W, m["heads"] * m["vdim"])
        vec(p + "mix.right.norm", m["heads"] * m["vdim"], 1.0)
        for t, b in (("i", 0.0), ("f", 2.0)):
            mat(p + "mix.right." + t, m["heads"], W)
            vec(p + f"mix.right.{t}.b", m["heads"], b, 1.0)
        vec(p + "mix.right.out", W, 1.0)
        if l["mlp"]:
            vec(p + "norm2", W, 0.0)
            mat(p + "mlp.up", l["mlp"]["ff"], W)
            mat(p + "mlp.down", W, l["mlp"]["ff"])
    vec("final.norm", W, 0.0)
    mat("head", cfg["vocab"], W, 2.0)
    return w


def write_folder(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    index, data, at = {}, [], 0
    for name, a in w.items():
        b = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        index[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        data.append(b)
    text = json.dumps(index).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(data))
    return path


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def want(cfg, w, toks):
    return L.forward(cfg, w, toks)


def rel(got, ref):
    """Per-row rms of the difference over the rms of all reference logits."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return np.sqrt(np.mean((got - ref) ** 2, axis=-1)) / np.sqrt(np.mean(ref ** 2))
