"""Small random Kuzipel models for the parity tests: configurations, weights, folders."""
from __future__ import annotations

import numpy as np

from oracle import layered as L
from tests.layered_util import bf16, rel, tokens, want, write_folder  # noqa: F401


def latent(heads, dim, rot, vdim, q_rank, kv_rank, scale=None, base=10000.0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}}}


def wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "rank": rank}      # the rank shows in a tensor only


def moe(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def config(width, vocab, eps, layers, mult=0.7, loop=None):
    c = {"architecture": "Kuzipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# Sizes that no tile divides, unequal layers, layers without feed-forward, one head, one expert, every expert, loops
# over the first layers, over the last ones, over everything and once only, heads too wide for the tensor-core kernel.
CONFIGS = {
    "mixed": config(88, 97, 1e-5, [layer(latent(5, 24, 12, 40, 36, 52), moe(6, 2, 40, 72)), layer(wkv(3, 24, 10), moe(5, 3, 33, 17)),
                                   layer(latent(2, 70, 6, 9, 20, 100), None), layer(wkv(2, 40, 5), None)], loop=(1, 3, 2)),
    "loop_first": config(64, 61, 1e-6, [layer(wkv(1, 32, 16), moe(4, 1, 24, 24)), layer(latent(1, 16, 2, 16, 8, 8), moe(3, 3, 16, 8))], 1.0, (0, 1, 3)),
    "loop_all": config(72, 70, 1e-3, [layer(latent(4, 16, 16, 16, 64, 64), None), layer(wkv(4, 16, 64), moe(9, 4, 20, 65))], 0.3, (0, 2, 2)),
    "once": config(75, 53, 1e-5, [layer(wkv(5, 7, 3), moe(2, 2, 31, 5)), layer(latent(3, 9, 4, 11, 13, 15), moe(12, 5, 7, 70))], 0.5, (1, 2, 1)),
    "no_loop": config(136, 83, 1e-5, [layer(wkv(1, 130, 33), None), layer(latent(2, 136, 24, 144, 90, 200), moe(4, 2, 130, 66)),
                                      layer(wkv(2, 65, 7), None)]),
    "wide": config(64, 40, 1e-5, [layer(latent(3, 264, 8, 12, 24, 40), None), layer(latent(33, 8, 8, 8, 24, 16), None),
                                  layer(latent(2, 8, 8, 264, 24, 16), None)]),
}


def weights(cfg, seed=0, steady=False):
    """name -> fp32 array holding bf16 values.  With `steady` the router's logits are far apart whatever a layer
    computes: some channels of the residual keep each token's own levels, and the router reads only those, so that
    rounding cannot change a choice."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    w = {}

    def mat(name, r, c, s=1.0):
        w[name] = bf16(s * rng.standard_normal((r, c)) / np.sqrt(c))

    def vec(name, n, mean, s=0.3):
        w[name] = bf16(mean + s * rng.standard_normal(n))

    kept = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"]], default=0) if steady else 0
    w["embed"] = bf16(0.5 + 1.5 * rng.standard_normal((cfg["vocab"], W)))
    for t in range(cfg["vocab"] if kept else 0):
        w["embed"][t, :kept] = bf16(rng.permutation(kept) * 1.0 - 0.5 * kept)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for k in ("1", "2") if l["mlp"] else ("1",):
            vec(p + "norm" + k, W, 1.0)
            vec(p + "ls" + k, W, 0.8, 0.4)
            if kept:
                w[p + "norm" + k][:kept] = 1.0
                w[p + "ls" + k][:kept] = 0.0
        p += "mix."
        if l["type"] == "latent_attention":
            H = m["heads"]
            mat(p + "dq", m["q_rank"], W)
            vec(p + "dq.norm", m["q_rank"], 1.0)
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + "dkv.norm", m["kv_rank"], 1.0)
            mat(p + "uk", H * m["dim"], m["kv_rank"], 1.5)
            mat(p + "uv", H * m["vdim"], m["kv_rank"])
            mat(p + "o", W, H * m["vdim"], 1.5)
        else:
            H, D, n = m["heads"], m["dim"], m["heads"] * m["dim"]
            for t in "rkvgw":
                w[p + "mu." + t] = bf16(rng.uniform(0, 1, W))
            for t in "rkvg":
                mat(p + t, n, W)
            mat(p + "w1", l["rank"], W)
            mat(p + "w2", n, l["rank"], 1.5)
            vec(p + "w0", n, -2.0, 2.0)
            w[p + "u"] = bf16(rng.standard_normal((H, D)))
            vec(p + "norm", n, 1.0)
            mat(p + "o", W, n, 1.5)
        if l["mlp"]:
            p, e = f"l{i}.mlp.", l["mlp"]
            E = e["router"]["experts"]
            for x in range(E):
                mat(p + f"e{x}.gate", e["expert"]["ff"], W, 1.5)
                mat(p + f"e{x}.up", e["expert"]["ff"], W, 1.5)
                mat(p + f"e{x}.down", W, e["expert"]["ff"], 2.0)
            if kept:
                w[p + "router"] = bf16(np.concatenate([np.eye(E), np.zeros((E, W - E))], 1))
                w[p + "router.b"] = bf16(0.05 * rng.standard_normal(E))
            else:
                mat(p + "router", E, W, 1.5)
                vec(p + "router.b", E, 0.0, 0.5)
            mat(p + "shared.gate", e["shared"]["ff"], W, 1.5)
            mat(p + "shared.up", e["shared"]["ff"], W, 1.5)
            mat(p + "shared.down", W, e["shared"]["ff"], 2.0)
            mat(p + "shared.sg", 1, W)
    if cfg.get("loop"):
        mat("loop.in", W, 2 * W)
        if kept:
            w["loop.in"][:kept] = 0
            w["loop.in"][:kept, :kept] = np.eye(kept)
    vec("final.norm", W, 1.0)
    mat("head", cfg["vocab"], W, 2.0)
    return w


def margin(cfg, w, toks):
    """The smallest distance between a chosen and a dropped router logit, over all tokens and layers."""
    least, route = [np.inf], L.route

    def watch(z, top):
        s = -np.sort(-z, axis=1)
        if top < z.shape[1]:
            least[0] = min(least[0], float((s[:, top - 1] - s[:, top]).min()))
        return route(z, top)

    L.route = watch
    try:
        L.forward(cfg, w, toks)
    finally:
        L.route = route
    return least[0]
