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

from .configs import CONFIGS, ModelConfig
from .layered import (MATH, EMBED, FINAL_NORM, HEAD, LAYER_SLOTS, SLOTS, GateAttention, LayeredConfig, LayeredInference,
                      MatrixMemory, ParallelLayer, slot_shapes)
from .safetensors import SafeTensors


class ConfigError(ValueError):
    pass


@dataclass(frozen=True)
class Architecture:
    name: str
    family: str                                     # library family that serves it (build.FAMILIES)
    read_config: Callable[[dict], object]           # config.json -> configuration
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


register(Architecture("Mitotar", "layered", mitotar_config, mitotar_weights))


# ---- loading ----------------------------------------------------------------------------------------

def read_config(folder: str):
    """(architecture, configuration) of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        j = json.load(f)
    name = j.get("architecture") or (j.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ConfigError(f"{folder}: architecture {name!r} is not registered (known: {', '.join(sorted(ARCHITECTURES))})")
    arch = ARCHITECTURES[name]
    return arch, arch.read_config(j)


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
