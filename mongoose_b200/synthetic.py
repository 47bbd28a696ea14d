"""Seeded synthetic models for the decode-path configurations.

The reference's published runs use public checkpoints that cannot be fetched
here; these generators stand in for them with the same shapes, block sizes
and an N(0, 0.02) weight distribution.  Everything is derived from
``numpy.random.default_rng`` seeds so that every consumer (engine, tests,
benchmark) sees identical tensors.
"""
from __future__ import annotations

import numpy as np

from . import configs as mc
from .layered import (NORM_LAYER, POS_NONE, GateAttention, LatentAttention, LayeredConfig, Loop, MatrixMemory, MixtureOfExperts,
                      ParallelLayer, PrenormLayer, Wkv, slot_shapes)
from .safetensors import to_bf16_bits


def single_matvec_case(seed: int = 0, N: int = 4864, K: int = 896):
    """One Q8_0 dequant-matvec: int8 blocks uniform in [-127,127], fp16 block
    scales |N(0,1)|*0.02/127, x ~ N(0,1).  Returns (raw blocks uint8 [N, K/32*34], x)."""
    rng = np.random.default_rng(seed)
    nb = K // 32
    q = rng.integers(-127, 128, size=(N, nb, 32), dtype=np.int8)
    d = (np.abs(rng.standard_normal((N, nb))) * 0.02 / 127.0).astype(np.float16)
    x = rng.standard_normal(K).astype(np.float32)
    blocks = np.empty((N, nb, 34), np.uint8)
    blocks[:, :, :2] = d.view(np.uint8).reshape(N, nb, 2)
    blocks[:, :, 2:] = q.view(np.uint8)
    return blocks.reshape(N, nb * 34), x


def tensor_f32(seed: int, idx: int, rows: int, cols: int, std: float = 0.02) -> np.ndarray:
    """The fp32 matrix for weight slot ``idx`` of a random-init model."""
    rng = np.random.default_rng([seed, idx])
    w = rng.standard_normal((rows, cols), dtype=np.float32)
    w *= np.float32(std)
    return w


def model_slots(cfg: mc.ModelConfig):
    """Yield (idx, kind, rows, cols, fmt) for every weight slot that is set.
    kind is "norm" or "matrix"."""
    for l in range(cfg.n_layers):
        base = l * 12
        yield base + mc.SLOT_NORM1, "norm", 1, cfg.dim, None
        yield base + mc.SLOT_NORM2, "norm", 1, cfg.dim, None
        for s in mc.MATRIX_SLOTS:
            r, c = cfg.matrix_shape(s)
            yield base + s, "matrix", r, c, cfg.layer_fmt
    yield cfg.n_layers * 12, "norm", 1, cfg.dim, None
    yield cfg.n_layers * 12 + 1, "matrix", cfg.vocab, cfg.dim, cfg.head_fmt


def norm_vector(seed: int, idx: int, dim: int, jitter: float = 0.0) -> np.ndarray:
    """RMSNorm weights: ones (random-init), optionally perturbed so that a kernel
    which ignores the norm weight cannot pass a test."""
    if jitter == 0.0:
        return np.ones(dim, np.float32)
    rng = np.random.default_rng([seed, idx, 7])
    return (1.0 + jitter * rng.standard_normal(dim)).astype(np.float32)


def prompt_ids(seed: int, n: int, vocab: int) -> np.ndarray:
    rng = np.random.default_rng([seed, 1 << 20])
    return rng.integers(0, vocab, size=n, dtype=np.int64).astype(np.int32)


def load_engine(engine, cfg: mc.ModelConfig, seed: int = 0, jitter: float = 0.0, on_matrix=None) -> None:
    """SetWeight every slot of a random-init model.  ``on_matrix(idx, w, fmt)`` is
    called with each fp32 matrix before it is dropped (benchmarks use it to hand the
    same tensor to the CPU baseline)."""
    for idx, kind, rows, cols, fmt in model_slots(cfg):
        if kind == "norm":
            v = norm_vector(seed, idx, cols, jitter)
            engine.SetWeight(idx, v)
            if on_matrix is not None:
                on_matrix(idx, v, None)
            continue
        w = tensor_f32(seed, idx, rows, cols)
        engine.SetWeight(idx, w)
        if on_matrix is not None:
            on_matrix(idx, w, fmt)
        del w


# ---- layer-described models -----------------------------------------------------------------------

def mitotar_like(name: str, width: int, n_layers: int, ffn: int, vocab: int, heads: int, kv_heads: int, dim: int, mem_heads: int,
                 mem_dim: int, max_seq: int) -> LayeredConfig:
    layer = ParallelLayer(GateAttention(heads, kv_heads, dim, dim ** -0.5, 0.25, 512), MatrixMemory(mem_heads, mem_dim, mem_dim, 15.0), ffn)
    return LayeredConfig(name=name, width=width, vocab=vocab, layers=(layer,) * n_layers, norm_eps=1e-6, max_seq=max_seq)


def kuzipel_like(name: str, width: int, n_layers: int, vocab: int, attn: LatentAttention, wkv: Wkv, moe: MixtureOfExperts,
                 max_seq: int) -> LayeredConfig:
    """`n_layers` layer runs: one attention layer, then two recurrent ones, and so on, the first recurrent one twice."""
    layers = tuple(PrenormLayer(wkv if i % 3 else attn, moe) for i in range(n_layers - 1))
    return LayeredConfig(name=name, width=width, vocab=vocab, layers=layers, norm_eps=1e-5, max_seq=max_seq, norm=NORM_LAYER,
                         positions=POS_NONE, residual_mult=0.5, loop=Loop(1, 2, 2))


def latent_like(heads: int, dim: int, rot_dim: int, q_rank: int, kv_rank: int) -> LatentAttention:
    return LatentAttention(heads, dim, rot_dim, dim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, 10000.0)


# layer widths of the dense configurations of the same name; a token's experts together are as wide as their feed-forward
LAYERED = {c.name: c for c in (
    mitotar_like("mitotar-tiny", 96, 2, 160, 300, 4, 2, 24, 3, 20, 256),
    mitotar_like("mitotar-0.5b", 896, 24, 4864, 151936, 14, 2, 64, 4, 128, 4096),
    mitotar_like("mitotar-1.1b", 2048, 22, 5632, 32000, 32, 4, 64, 8, 128, 4096),
    mitotar_like("mitotar-7b-width-4l", 3584, 4, 18944, 16000, 28, 4, 128, 8, 256, 4096),
    kuzipel_like("kuzipel-tiny", 96, 5, 300, latent_like(3, 24, 8, 40, 56), Wkv(4, 20, 12), MixtureOfExperts(5, 2, 40, 72), 256),
    kuzipel_like("kuzipel-0.5b", 896, 24, 151936, latent_like(14, 64, 32, 384, 256), Wkv(14, 64, 64), MixtureOfExperts(16, 4, 608, 2432), 4096),
    kuzipel_like("kuzipel-1.1b", 2048, 22, 32000, latent_like(16, 128, 64, 768, 512), Wkv(32, 64, 64), MixtureOfExperts(16, 4, 704, 2816), 4096),
    kuzipel_like("kuzipel-7b-width-4l", 3584, 4, 16000, latent_like(28, 128, 64, 1536, 512), Wkv(56, 64, 64),
                 MixtureOfExperts(16, 4, 2368, 9472), 4096),
)}


def layered_tensors(cfg: LayeredConfig, seed: int = 0):
    """Yield (slot, name, layer, fp32 tensor) of a random-init model: matrices N(0, 1 / fan-in), head mixing
    near the identity, norm weights and biases jittered around their neutral value."""
    around_zero = {"at.bias", "mem.i_bias", "moe.bias"} | ({"norm1", "norm2", "final_norm"} if cfg.norm != NORM_LAYER else set())
    for idx, name, layer, rows, cols in slot_shapes(cfg):
        rng = np.random.default_rng([seed, idx])
        if rows:
            w = rng.standard_normal((rows, cols), dtype=np.float32)
            w *= np.float32(1.0 if name == "embed" else cols ** -0.5)
        elif name == "at.talk":
            n = cfg.layers[layer].attn.heads
            w = (np.eye(n) + 0.3 * n ** -0.5 * rng.standard_normal((n, n))).astype(np.float32).reshape(-1)
        else:
            neutral = 0.0 if name in around_zero else 3.0 if name == "mem.f_bias" else -2.0 if name == "wkv.w0" else 0.5 if "mu_" in name else 1.0
            w = (neutral + 0.2 * rng.standard_normal(cols)).astype(np.float32)
        yield idx, name, layer, w


def load_layered(engine, seed: int = 0, on_tensor=None) -> None:
    """Random-init weights for every slot of a layer-described model."""
    for idx, name, layer, w in layered_tensors(engine.cfg, seed):
        bits = to_bf16_bits(w)
        engine.SetWeightBF16(idx, bits)
        if on_tensor is not None:
            on_tensor(name, layer, bits)
    engine.BuildFusedDispatch()
