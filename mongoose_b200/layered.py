"""Models described layer by layer: configuration, weight slots and engine.

A configuration lists its layers one by one (mixer, feed-forward, sizes); ``LayeredInference`` builds
the engine for it and inherits every stepping call of ``CUDAFusedInference`` (StepToken, Generate,
PartialStep, cursor, introspection), because both are handles of the same C++ engine.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, replace
from typing import Iterator

import numpy as np

from . import _lib
from .configs import FMT_BF16
from .fused_infer import CUDAFusedInference, MongooseError, _np_ptr

MATH_BF16, MATH_F32 = 0, 1
MATH = {"bfloat16": MATH_BF16, "float32": MATH_F32}
MIXER_PARALLEL = 0

# weight slots within a layer (MG_SLOT_* of include/mongoose_kernels.h)
LAYER_SLOTS = 32
SLOTS = {
    "norm1": 0, "norm2": 1,
    "at.q": 2, "at.k": 3, "at.q_norm": 4, "at.k_norm": 5, "at.talk": 6, "at.bias": 7, "at.o": 8, "at.out": 9,
    "mem.q": 10, "mem.k": 11, "mem.v": 12, "mem.g": 13, "mem.o": 14, "mem.norm": 15,
    "mem.i": 16, "mem.i_bias": 17, "mem.f": 18, "mem.f_bias": 19, "mem.out": 20,
    "up": 21, "down": 22,
}
EMBED, FINAL_NORM, HEAD = 0, 1, 2       # after the layers


@dataclass(frozen=True)
class GateAttention:
    """Sigmoid attention with mixed heads; the values are the raw keys."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 1


@dataclass(frozen=True)
class MatrixMemory:
    """Per-head [dim, vdim] state with capped exponential gates."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelLayer:
    attn: GateAttention
    mem: MatrixMemory
    ffn_dim: int = 0            # 0: no feed-forward


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    width: int
    vocab: int
    layers: tuple[ParallelLayer, ...]
    norm_eps: float
    max_seq: int = 1024
    math: int = MATH_BF16

    def with_(self, **kw) -> "LayeredConfig":
        return replace(self, **kw)

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def dim(self) -> int:
        return self.width


def slot_shapes(cfg: LayeredConfig) -> Iterator[tuple[int, str, int, int, int]]:
    """(slot index, slot name, layer or -1, rows, cols) of every weight; vectors have 0 rows."""
    W = cfg.width
    for i, l in enumerate(cfg.layers):
        a, m = l.attn, l.mem
        shapes = {
            "norm1": (0, W), "at.q": (a.heads * a.dim, W), "at.k": (a.kv_heads * a.dim, W),
            "at.q_norm": (0, a.dim), "at.k_norm": (0, a.dim), "at.talk": (0, a.heads * a.heads), "at.bias": (0, a.heads),
            "at.o": (W, a.heads * a.dim), "at.out": (0, W),
            "mem.q": (m.heads * m.dim, W), "mem.k": (m.heads * m.dim, W), "mem.v": (m.heads * m.vdim, W),
            "mem.g": (m.heads * m.vdim, W), "mem.o": (W, m.heads * m.vdim), "mem.norm": (0, m.heads * m.vdim),
            "mem.i": (m.heads, W), "mem.i_bias": (0, m.heads), "mem.f": (m.heads, W), "mem.f_bias": (0, m.heads),
            "mem.out": (0, W),
        }
        if l.ffn_dim:
            shapes.update({"norm2": (0, W), "up": (l.ffn_dim, W), "down": (W, l.ffn_dim)})
        for name, (r, c) in shapes.items():
            yield i * LAYER_SLOTS + SLOTS[name], name, i, r, c
    base = cfg.n_layers * LAYER_SLOTS
    yield base + EMBED, "embed", -1, cfg.vocab, W
    yield base + FINAL_NORM, "final_norm", -1, 0, W
    yield base + HEAD, "head", -1, cfg.vocab, W


def weight_bytes_per_token(cfg: LayeredConfig) -> int:
    """bf16 bytes of the matrices one decode token streams (every layer matrix and the head)."""
    return sum(2 * r * c for _, name, _, r, c in slot_shapes(cfg) if r and name != "embed")


def cache_bytes_per_position(cfg: LayeredConfig) -> int:
    """Cached keys (raw rows and their 1 / rms) one position adds to what a decode token reads."""
    eb = 4 if cfg.math == MATH_F32 else 2
    return sum(l.attn.kv_heads * (-(-l.attn.dim // 8) * 8 * eb + 4) for l in cfg.layers)


def state_bytes(cfg: LayeredConfig) -> int:
    """Recurrent state one decode token reads (and writes again)."""
    return sum(4 * l.mem.heads * (l.mem.dim * (l.mem.vdim + 1) + 1) for l in cfg.layers)


def prefill_flops(cfg: LayeredConfig, n: int) -> float:
    """Multiply-adds x 2 of a prompt of n tokens from position 0: matrices, causal scores, head mixing and
    values, and the recurrence of the memory."""
    total = 0.0
    for l in cfg.layers:
        a, m, W = l.attn, l.mem, cfg.width
        total += n * W * (2 * a.heads * a.dim + a.kv_heads * a.dim + m.heads * (2 * m.dim + 3 * m.vdim + 2) + 2 * l.ffn_dim)
        total += n * (n + 1) / 2 * a.heads * (2 * a.dim + a.heads)
        total += n * m.heads * 2 * m.dim * m.vdim
    return 2.0 * total


class LayeredInference(CUDAFusedInference):
    def __init__(self, cfg: LayeredConfig, device: int = 0):
        self.cfg = cfg
        self._lib = _lib.load(family="layered")
        c = _lib.MgModelConfig(width=cfg.width, vocab=cfg.vocab, n_layers=cfg.n_layers, max_seq=cfg.max_seq,
                               norm_eps=cfg.norm_eps, math=cfg.math, device=device)
        ls = (_lib.MgLayerConfig * cfg.n_layers)()
        for d, l in zip(ls, cfg.layers):
            d.mixer = MIXER_PARALLEL
            d.attn = _lib.MgGateAttnConfig(l.attn.heads, l.attn.kv_heads, l.attn.dim, l.attn.scale, l.attn.temp_coef, l.attn.temp_every)
            d.mem = _lib.MgMatMemConfig(l.mem.heads, l.mem.dim, l.mem.vdim, l.mem.gate_cap)
            d.ffn_dim = l.ffn_dim
        h = C.c_void_p()
        rc = self._lib.mg_create_layered(C.byref(c), ls, C.byref(h))
        if rc != 0 or not h.value:
            raise MongooseError(f"mg_create_layered failed with status {rc} (is a B200 visible as device {device}?)")
        self._h = h
        self.tp_rank, self.tp_size = 0, 1

    def SetWeightBF16(self, idx: int, bits) -> None:
        """bf16 bit patterns (uint16) for any slot; norms and biases are widened exactly."""
        a = np.ascontiguousarray(bits, dtype=np.uint16)
        self._check(self._lib.mg_set_weight_raw(self._h, idx, _np_ptr(a), a.nbytes, FMT_BF16), f"SetWeightBF16({idx})")
