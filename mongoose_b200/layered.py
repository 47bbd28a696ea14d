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
MIXER_PARALLEL, MIXER_LATENT, MIXER_WKV = 0, 1, 2
NORM_RMS_AROUND_ZERO, NORM_LAYER, NORM_RMS = 0, 1, 2
POS_SINUSOID, POS_NONE = 0, 1

# weight slots within a layer (MG_SLOT_* of include/mongoose_kernels.h)
LAYER_SLOTS = 64
SLOTS = {
    "norm1": 0, "norm2": 1,
    "at.q": 2, "at.k": 3, "at.q_norm": 4, "at.k_norm": 5, "at.talk": 6, "at.bias": 7, "at.o": 8, "at.out": 9,
    "mem.q": 10, "mem.k": 11, "mem.v": 12, "mem.g": 13, "mem.o": 14, "mem.norm": 15,
    "mem.i": 16, "mem.i_bias": 17, "mem.f": 18, "mem.f_bias": 19, "mem.out": 20,
    "up": 21, "down": 22, "ls1": 23, "ls2": 24,
    "la.dq": 25, "la.dq_norm": 26, "la.uq": 27, "la.dkv": 28, "la.dkv_norm": 29, "la.uk": 30, "la.uv": 31, "la.o": 32,
    "wkv.mu_r": 33, "wkv.mu_k": 34, "wkv.mu_v": 35, "wkv.mu_g": 36, "wkv.mu_w": 37,
    "wkv.r": 38, "wkv.k": 39, "wkv.v": 40, "wkv.g": 41, "wkv.w1": 42, "wkv.w2": 43, "wkv.w0": 44, "wkv.u": 45, "wkv.norm": 46, "wkv.o": 47,
    "moe.router": 48, "moe.bias": 49, "moe.gate": 50, "moe.up": 51, "moe.down": 52,
    "shared.gate": 53, "shared.up": 54, "shared.down": 55, "shared.sg": 56,
}
EMBED, FINAL_NORM, HEAD, LOOP_IN = 0, 1, 2, 3       # after the layers


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
class LatentAttention:
    """Softmax attention over a cached low-rank latent and one rotated key part for all heads."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass(frozen=True)
class Wkv:
    """Per-head [dim, dim] state with a data-dependent decay per key channel, on token-shifted inputs."""
    heads: int
    dim: int
    decay_rank: int


@dataclass(frozen=True)
class MixtureOfExperts:
    """`top` of `experts` gated feed-forwards per token, and a shared one (shared_ff = 0: none)."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0


@dataclass(frozen=True)
class PrenormLayer:
    mixer: LatentAttention | Wkv
    moe: MixtureOfExperts | None = None


@dataclass(frozen=True)
class Loop:
    """Layers start .. stop - 1 run `times` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    width: int
    vocab: int
    layers: tuple[ParallelLayer | PrenormLayer, ...]
    norm_eps: float
    max_seq: int = 1024
    math: int = MATH_BF16
    norm: int = NORM_RMS_AROUND_ZERO
    positions: int = POS_SINUSOID
    residual_mult: float = 1.0
    loop: Loop | None = None

    def with_(self, **kw) -> "LayeredConfig":
        return replace(self, **kw)

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def dim(self) -> int:
        return self.width

    def runs(self) -> tuple[int, ...]:
        """Layer index of every layer run, in order; the stepping calls count these."""
        if not self.loop:
            return tuple(range(self.n_layers))
        a, b = self.loop.start, self.loop.stop
        return (*range(a), *(tuple(range(a, b)) * self.loop.times), *range(b, self.n_layers))


def _parallel_shapes(l: ParallelLayer, W: int) -> dict[str, tuple[int, int]]:
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
    return shapes


def _prenorm_shapes(l: PrenormLayer, W: int) -> dict[str, tuple[int, int]]:
    m, e = l.mixer, l.moe
    shapes = {"norm1": (0, W), "ls1": (0, W)}
    if isinstance(m, LatentAttention):
        shapes.update({
            "la.dq": (m.q_rank, W), "la.dq_norm": (0, m.q_rank), "la.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
            "la.dkv": (m.kv_rank + m.rot_dim, W), "la.dkv_norm": (0, m.kv_rank), "la.uk": (m.heads * m.dim, m.kv_rank),
            "la.uv": (m.heads * m.vdim, m.kv_rank), "la.o": (W, m.heads * m.vdim)})
    else:
        n = m.heads * m.dim
        shapes.update({"wkv.mu_" + t: (0, W) for t in "rkvgw"})
        shapes.update({"wkv." + t: (n, W) for t in "rkvg"})
        shapes.update({"wkv.w1": (m.decay_rank, W), "wkv.w2": (n, m.decay_rank), "wkv.w0": (0, n), "wkv.u": (0, n), "wkv.norm": (0, n),
                       "wkv.o": (W, n)})
    if e:
        shapes.update({"norm2": (0, W), "ls2": (0, W), "moe.router": (e.experts, W), "moe.bias": (0, e.experts),
                       "moe.gate": (e.experts * e.ff, W), "moe.up": (e.experts * e.ff, W), "moe.down": (e.experts * W, e.ff)})
        if e.shared_ff:
            shapes.update({"shared.gate": (e.shared_ff, W), "shared.up": (e.shared_ff, W), "shared.down": (W, e.shared_ff), "shared.sg": (1, W)})
    return shapes


def slot_shapes(cfg: LayeredConfig) -> Iterator[tuple[int, str, int, int, int]]:
    """(slot index, slot name, layer or -1, rows, cols) of every weight; vectors have 0 rows."""
    W = cfg.width
    for i, l in enumerate(cfg.layers):
        for name, (r, c) in (_parallel_shapes if isinstance(l, ParallelLayer) else _prenorm_shapes)(l, W).items():
            yield i * LAYER_SLOTS + SLOTS[name], name, i, r, c
    base = cfg.n_layers * LAYER_SLOTS
    yield base + EMBED, "embed", -1, cfg.vocab, W
    yield base + FINAL_NORM, "final_norm", -1, 0, W
    yield base + HEAD, "head", -1, cfg.vocab, W
    if cfg.loop:
        yield base + LOOP_IN, "loop_in", -1, W, 2 * W


def weight_bytes_per_token(cfg: LayeredConfig) -> int:
    """bf16 bytes of the matrices one decode token streams (every layer run's matrices, the chosen experts
    among them, and the head)."""
    runs, total = cfg.runs(), 0
    for _, name, layer, r, c in slot_shapes(cfg):
        if not r or name == "embed":
            continue
        share = 1.0
        if name in ("moe.gate", "moe.up", "moe.down"):
            share = cfg.layers[layer].moe.top / cfg.layers[layer].moe.experts
        times = runs.count(layer) if layer >= 0 else cfg.loop.times if name == "loop_in" else 1
        total += round(2 * r * c * share) * times
    return total


def cache_bytes_per_position(cfg: LayeredConfig) -> int:
    """Cached bytes one position adds to what a decode token reads: raw key rows and their 1 / rms, or the
    latent and the rotated key part."""
    eb = 4 if cfg.math == MATH_F32 else 2
    total = 0
    for i in cfg.runs():
        l = cfg.layers[i]
        if isinstance(l, ParallelLayer):
            total += l.attn.kv_heads * (-(-l.attn.dim // 8) * 8 * eb + 4)
        elif isinstance(l.mixer, LatentAttention):
            total += (-(-l.mixer.kv_rank // 8) + -(-l.mixer.rot_dim // 8)) * 8 * eb
    return total


def state_bytes(cfg: LayeredConfig) -> int:
    """Recurrent state one decode token reads (and writes again)."""
    total = 0
    for i in cfg.runs():
        l = cfg.layers[i]
        if isinstance(l, ParallelLayer):
            total += 4 * l.mem.heads * (l.mem.dim * (l.mem.vdim + 1) + 1)
        elif isinstance(l.mixer, Wkv):
            total += 4 * (l.mixer.heads * l.mixer.dim ** 2 + cfg.width)
    return total


def prefill_flops(cfg: LayeredConfig, n: int) -> float:
    """Multiply-adds x 2 of a prompt of n tokens from position 0: matrices, causal scores, head mixing and
    values, and the recurrences."""
    total, W = 0.0, cfg.width
    for i in cfg.runs():
        l = cfg.layers[i]
        if isinstance(l, ParallelLayer):
            a, m = l.attn, l.mem
            total += n * W * (2 * a.heads * a.dim + a.kv_heads * a.dim + m.heads * (2 * m.dim + 3 * m.vdim + 2) + 2 * l.ffn_dim)
            total += n * (n + 1) / 2 * a.heads * (2 * a.dim + a.heads)
            total += n * m.heads * 2 * m.dim * m.vdim
            continue
        m, e = l.mixer, l.moe
        if isinstance(m, LatentAttention):
            total += n * (W * (m.q_rank + m.kv_rank + m.rot_dim + m.heads * m.vdim) + m.q_rank * m.heads * (m.dim + m.rot_dim) +
                          m.kv_rank * m.heads * (m.dim + m.vdim))
            total += n * (n + 1) / 2 * m.heads * (m.dim + m.rot_dim + m.vdim)
        else:
            total += n * (W * (5 * m.heads * m.dim + m.decay_rank) + m.decay_rank * m.heads * m.dim + 2 * m.heads * m.dim ** 2)
        if e:
            total += n * W * (e.experts + 3 * e.top * e.ff + 3 * e.shared_ff + (1 if e.shared_ff else 0))
    if cfg.loop:
        total += n * 2 * W * W * cfg.loop.times
    return 2.0 * total


class LayeredInference(CUDAFusedInference):
    def __init__(self, cfg: LayeredConfig, device: int = 0):
        self.cfg = cfg
        self._lib = _lib.load(family="layered")
        c = _lib.MgModelConfig(width=cfg.width, vocab=cfg.vocab, n_layers=cfg.n_layers, max_seq=cfg.max_seq,
                               norm_eps=cfg.norm_eps, math=cfg.math, device=device, norm=cfg.norm, positions=cfg.positions,
                               residual_mult=cfg.residual_mult)
        if cfg.loop:
            c.loop_start, c.loop_stop, c.loop_times = cfg.loop.start, cfg.loop.stop, cfg.loop.times
        ls = (_lib.MgLayerConfig * cfg.n_layers)()
        for d, l in zip(ls, cfg.layers):
            if isinstance(l, ParallelLayer):
                d.mixer = MIXER_PARALLEL
                d.attn = _lib.MgGateAttnConfig(l.attn.heads, l.attn.kv_heads, l.attn.dim, l.attn.scale, l.attn.temp_coef, l.attn.temp_every)
                d.mem = _lib.MgMatMemConfig(l.mem.heads, l.mem.dim, l.mem.vdim, l.mem.gate_cap)
                d.ffn_dim = l.ffn_dim
                continue
            m, e = l.mixer, l.moe
            if isinstance(m, LatentAttention):
                d.mixer = MIXER_LATENT
                d.latent = _lib.MgLatentAttnConfig(m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_base)
            else:
                d.mixer = MIXER_WKV
                d.wkv = _lib.MgWkvConfig(m.heads, m.dim, m.decay_rank)
            if e:
                d.moe = _lib.MgMoeConfig(e.experts, e.top, e.ff, e.shared_ff)
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
