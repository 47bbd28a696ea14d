"""Model registry: which class serves a model, and how a model folder is read.

Two kinds of entries: named configurations (the dense decode block, random-init weights from
``synthetic``), and architectures that are loaded from a folder with ``config.json`` and
``model.safetensors``; ``config.json``'s "architecture" names the entry.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

import numpy as np

from .configs import CONFIGS, ModelConfig
from .layered import (MATH, NORM_LAYER, POS_NONE, GateAttention, LatentAttention, LayeredConfig, LayeredInference, Loop,
                      MatrixMemory, MixtureOfExperts, ParallelLayer, PrenormLayer, Wkv, slot_shapes)
from .safetensors import SafeTensors


class ConfigError(ValueError):
    pass


@dataclass(frozen=True)
class Architecture:
    name: str
    family: str                                     # library family that serves it (build.FAMILIES)
    # config.json, and a function that gives a tensor's shape -> configuration
    read_config: Callable[[dict, Callable[[str], tuple[int, ...]]], object]
    load_weights: Callable[[object, SafeTensors], None]


ARCHITECTURES: dict[str, Architecture] = {}


def register(arch: Architecture) -> None:
    ARCHITECTURES[arch.name] = arch


def _get(d: dict, key: str, where: str):
    if key not in d:
        raise ConfigError(f"{where}: {key!r} is missing")
    return d[key]


# ---- Mitotar --------------------------------------------------------------------------------------

def mitotar_config(j: dict) -> LayeredConfig:
    layers = []
    for i, l in enumerate(_get(j, "layers", "config")):
        where = f"layer {i}"
        if _get(l, "type", where) != "parallel":
            raise ConfigError(f"{where}: mixer type {l['type']!r} is not known")
        mix = _get(l, "mixer", where)
        a, m = _get(mix, "left", where), _get(mix, "right", where)
        if a.get("vdim", a["dim"]) != a["dim"]:
            raise ConfigError(f"{where}: the values are the keys, but vdim {a['vdim']} differs from dim {a['dim']}")
        temp = a.get("q_temp") or {"coef": 0.0, "every": 1}
        if int(temp["every"]) != temp["every"] or temp["every"] < 1:
            raise ConfigError(f"{where}: q_temp.every must be a positive whole number")
        mlp = l.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ConfigError(f"{where}: feed-forward kind {mlp['kind']!r} is not known")
        layers.append(ParallelLayer(
            GateAttention(heads=_get(a, "heads", where), kv_heads=a.get("kv_heads", a["heads"]), dim=_get(a, "dim", where),
                          scale=float(_get(a, "scale", where)), temp_coef=float(temp["coef"]), temp_every=int(temp["every"])),
            MatrixMemory(heads=_get(m, "heads", where), dim=_get(m, "dim", where), vdim=m.get("vdim", m["dim"]),
                         gate_cap=float(_get(m, "gate_cap", where))),
            int(mlp["ff"]) if mlp else 0))
    return LayeredConfig(name="Mitotar", width=_get(j, "width", "config"), vocab=_get(j, "vocab", "config"), layers=tuple(layers),
                         norm_eps=float(_get(_get(j, "norm", "config"), "eps", "norm")))


# slot -> tensor name under the layer's prefix
MITOTAR_TENSORS = {
    "norm1": "norm1", "norm2": "norm2",
    "at.q": "mix.left.q", "at.k": "mix.left.k", "at.q_norm": "mix.left.q.norm", "at.k_norm": "mix.left.k.norm",
    "at.talk": "mix.left.talk", "at.bias": "mix.left.pb", "at.o": "mix.left.o", "at.out": "mix.left.out",
    "mem.q": "mix.right.q", "mem.k": "mix.right.k", "mem.v": "mix.right.v", "mem.g": "mix.right.g", "mem.o": "mix.right.o",
    "mem.norm": "mix.right.norm", "mem.i": "mix.right.i", "mem.i_bias": "mix.right.i.b", "mem.f": "mix.right.f",
    "mem.f_bias": "mix.right.f.b", "mem.out": "mix.right.out",
    "up": "mlp.up", "down": "mlp.down",
}
MITOTAR_GLOBALS = {"embed": "embed", "final_norm": "final.norm", "head": "head"}


def mitotar_tensor(slot_name: str, layer: int) -> str:
    return MITOTAR_GLOBALS[slot_name] if layer < 0 else f"l{layer}.{MITOTAR_TENSORS[slot_name]}"


def mitotar_weights(engine: LayeredInference, st: SafeTensors) -> None:
    for idx, name, layer, rows, cols in slot_shapes(engine.cfg):
        t = mitotar_tensor(name, layer)
        bits = st.bf16_bits(t)
        if bits.size != max(rows, 1) * cols or (rows and bits.shape != (rows, cols)):
            raise ConfigError(f"{t}: shape {bits.shape} does not fit the configuration ({rows} x {cols})")
        engine.SetWeightBF16(idx, bits)


register(Architecture("Mitotar", "layered", lambda j, shape: mitotar_config(j), mitotar_weights))


# ---- Kuzipel --------------------------------------------------------------------------------------

def kuzipel_config(j: dict, shape: Callable[[str], tuple[int, ...]]) -> LayeredConfig:
    """The rank of a recurrent layer's decay is known from its tensor only."""
    layers = []
    for i, l in enumerate(_get(j, "layers", "config")):
        where = f"layer {i}"
        kind, m = _get(l, "type", where), _get(l, "mixer", where)
        if kind == "latent_attention":
            rot = _get(m, "rot", where)
            rot_dim = int(_get(m, "rot_dim", where))
            if rot.get("dims", rot_dim) != rot_dim or rot_dim < 2 or rot_dim % 2:
                raise ConfigError(f"{where}: the rotated part has rot_dim {rot_dim} dimensions, rot.dims {rot.get('dims')} of them rotated")
            dim = int(_get(m, "dim", where))
            mixer = LatentAttention(heads=int(_get(m, "heads", where)), dim=dim, rot_dim=rot_dim, vdim=int(m.get("vdim", dim)),
                                    q_rank=int(_get(m, "q_rank", where)), kv_rank=int(_get(m, "kv_rank", where)),
                                    scale=float(_get(m, "scale", where)), rot_base=float(_get(rot, "base", where)))
        elif kind == "wkv":
            mixer = Wkv(heads=int(_get(m, "heads", where)), dim=int(_get(m, "dim", where)), decay_rank=int(shape(f"l{i}.mix.w1")[0]))
        else:
            raise ConfigError(f"{where}: mixer type {kind!r} is not known")
        mlp = l.get("mlp")
        moe = None
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ConfigError(f"{where}: feed-forward kind {mlp['kind']!r} is not known")
            router, shared = _get(mlp, "router", where), mlp.get("shared")
            moe = MixtureOfExperts(experts=int(_get(router, "experts", where)), top=int(_get(router, "top", where)),
                                   ff=int(_get(_get(mlp, "expert", where), "ff", where)), shared_ff=int(_get(shared, "ff", where)) if shared else 0)
            if not 1 <= moe.top <= moe.experts:
                raise ConfigError(f"{where}: {moe.top} of {moe.experts} experts cannot be chosen")
        layers.append(PrenormLayer(mixer, moe))
    loop = j.get("loop")
    if loop:
        loop = Loop(int(_get(loop, "start", "loop")), int(_get(loop, "stop", "loop")), int(_get(loop, "times", "loop")))
        if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
            raise ConfigError(f"loop: layers {loop.start} to {loop.stop} of {len(layers)}, {loop.times} times")
    return LayeredConfig(name="Kuzipel", width=int(_get(j, "width", "config")), vocab=int(_get(j, "vocab", "config")), layers=tuple(layers),
                         norm_eps=float(_get(_get(j, "norm", "config"), "eps", "norm")), norm=NORM_LAYER, positions=POS_NONE,
                         residual_mult=float(j.get("residual_mult", 1.0)), loop=loop or None)


# slot -> tensor name under the layer's prefix; {e} stands for an expert
KUZIPEL_TENSORS = {
    "norm1": "norm1", "norm2": "norm2", "ls1": "ls1", "ls2": "ls2",
    "la.dq": "mix.dq", "la.dq_norm": "mix.dq.norm", "la.uq": "mix.uq", "la.dkv": "mix.dkv", "la.dkv_norm": "mix.dkv.norm",
    "la.uk": "mix.uk", "la.uv": "mix.uv", "la.o": "mix.o",
    **{f"wkv.mu_{t}": f"mix.mu.{t}" for t in "rkvgw"},
    **{f"wkv.{t}": f"mix.{t}" for t in ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")},
    "moe.router": "mlp.router", "moe.bias": "mlp.router.b", "moe.gate": "mlp.e{e}.gate", "moe.up": "mlp.e{e}.up", "moe.down": "mlp.e{e}.down",
    "shared.gate": "mlp.shared.gate", "shared.up": "mlp.shared.up", "shared.down": "mlp.shared.down", "shared.sg": "mlp.shared.sg",
}
KUZIPEL_GLOBALS = {"embed": "embed", "final_norm": "final.norm", "head": "head", "loop_in": "loop.in"}


def kuzipel_tensors(cfg: LayeredConfig, slot_name: str, layer: int) -> list[str]:
    """The tensors a slot holds, stacked one below the other."""
    if layer < 0:
        return [KUZIPEL_GLOBALS[slot_name]]
    t = f"l{layer}.{KUZIPEL_TENSORS[slot_name]}"
    return [t.format(e=e) for e in range(cfg.layers[layer].moe.experts)] if "{e}" in t else [t]


def kuzipel_weights(engine: LayeredInference, st: SafeTensors) -> None:
    for idx, name, layer, rows, cols in slot_shapes(engine.cfg):
        names = kuzipel_tensors(engine.cfg, name, layer)
        parts = [st.bf16_bits(t) for t in names]
        for t, b in zip(names, parts):
            if (b.shape != (rows // len(names), cols)) if rows else (b.size != cols):
                raise ConfigError(f"{t}: shape {b.shape} does not fit the configuration ({rows // len(names)} x {cols})")
        engine.SetWeightBF16(idx, parts[0] if len(parts) == 1 else np.concatenate(parts))


register(Architecture("Kuzipel", "layered", kuzipel_config, kuzipel_weights))


# ---- loading ----------------------------------------------------------------------------------------

def read_config(folder: str):
    """(architecture, configuration) of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        j = json.load(f)
    name = j.get("architecture") or (j.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ConfigError(f"{folder}: architecture {name!r} is not registered (known: {', '.join(sorted(ARCHITECTURES))})")
    arch = ARCHITECTURES[name]
    weights: list[SafeTensors] = []

    def shape(tensor: str) -> tuple[int, ...]:
        if not weights:
            weights.append(SafeTensors(os.path.join(folder, "model.safetensors")))
        if tensor not in weights[0]:
            raise ConfigError(f"{folder}: no tensor {tensor!r}")
        return weights[0].shape(tensor)

    return arch, arch.read_config(j, shape)


def create_engine(cfg, device: int = 0):
    """The engine class that serves a configuration."""
    if isinstance(cfg, LayeredConfig):
        return LayeredInference(cfg, device=device)
    from .fused_infer import CUDAFusedInference
    return CUDAFusedInference(cfg, device=device)


def load_model(folder: str, dtype: str = "bfloat16", max_seq: int | None = None, device: int = 0):
    """Engine with the weights of a model folder, ready to step."""
    arch, cfg = read_config(folder)
    if dtype not in MATH:
        raise ConfigError(f"dtype {dtype!r}: one of {', '.join(MATH)}")
    cfg = cfg.with_(math=MATH[dtype], **({"max_seq": max_seq} if max_seq else {}))
    engine = create_engine(cfg, device)
    arch.load_weights(engine, SafeTensors(os.path.join(folder, "model.safetensors")))
    engine.BuildFusedDispatch()
    return engine


def named_config(name: str) -> ModelConfig | LayeredConfig:
    from . import synthetic
    if name in CONFIGS:
        return CONFIGS[name]
    if name in synthetic.LAYERED:
        return synthetic.LAYERED[name]
    raise ConfigError(f"no configuration {name!r} (known: {', '.join(sorted([*CONFIGS, *synthetic.LAYERED]))})")
