"""Goselix: a decoder whose layers run a mixer and a feed-forward side by side on the same stream, each
behind an RMS norm of its own.  Mixers are latent attention (queries, keys and values from low-rank latents;
the cache holds one latent and one rotated key part per token) and retention (a matrix state per head with a
fixed decay); feed-forwards are SiLU-gated, dense or a mixture of experts whose sigmoid scores scale what goes
into an expert.  A range of layers runs several times with the same weights, each pass with a step vector of
its own and, after the first, the embedding output added to the stream.

``load`` reads a folder with ``config.json`` and ``model.safetensors``; :class:`Goselix` lays the weights out
the way ``caten_b200_decoder_create`` takes them (include/caten_b200.h) and steps the model through it.  Every
size and constant comes from the configuration.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

import numpy as np

from . import _lib as L
from .decoder import DecoderModel, _head_cols, _head_rows, _pad, load_folder, p16, p64, rope_frequencies
from .runtime import B200Runtime
from .safetensors import bf16_to_f32

ARCHITECTURE = "Goselix"
CHUNK = 64   # tokens per chunk of a retention prompt: decay powers 0 .. CHUNK are tabulated


# ---- configuration ------------------------------------------------------------------------------
@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    rot_base: float
    scale: float


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    rot_dims: int
    rot_base: float
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[LatentConfig, RetentionConfig]
    mlp: Union[DenseConfig, ExpertsConfig, None]


@dataclass(frozen=True)
class GoselixConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerConfig, ...]
    loop: Optional[Tuple[int, int, int]]   # start, stop, times


def _latent(m: dict) -> LatentConfig:
    if int(m["rot"]["dims"]) != int(m["rot_dim"]):
        raise ValueError(f"rot.dims {m['rot']['dims']} is not rot_dim {m['rot_dim']}")
    return LatentConfig(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")), float(m["rot"]["base"]), float(m["scale"]))


def _retention(m: dict) -> RetentionConfig:
    decay = tuple(float(d) for d in m["decay"])
    if len(decay) != int(m["heads"]):
        raise ValueError(f"{len(decay)} decays for {m['heads']} heads")
    return RetentionConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["rot"]["dims"]), float(m["rot"]["base"]), decay)


def _dense(m: dict) -> DenseConfig:
    return DenseConfig(int(m["ff"]))


def _moe(m: dict) -> ExpertsConfig:
    e, top = int(m["router"]["experts"]), int(m["router"]["top"])
    if not 1 <= top <= e:
        raise ValueError(f"{top} of {e} experts")
    return ExpertsConfig(int(m["expert"]["ff"]), e, top)


_MIXERS = {"latent_attention": _latent, "retention": _retention}
_MLPS = {"dense": _dense, "moe": _moe}


def parse_config(cfg: dict) -> GoselixConfig:
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCHITECTURE}")
    layers = []
    for i, l in enumerate(cfg["layers"]):
        mlp = l.get("mlp")
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
        if mlp is not None and mlp["kind"] not in _MLPS:
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(LayerConfig(_MIXERS[l["type"]](l["mixer"]), _MLPS[mlp["kind"]](mlp) if mlp is not None else None))
    loop = cfg.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
    return GoselixConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]), tuple(layers), loop or None)


# ---- weight layout (bf16 bit patterns, padded with zeros) ------------------------------------------
def _head_parts(a: np.ndarray, heads: int, parts, cols: int) -> np.ndarray:
    """[heads * sum(parts), K] -> [heads * sum(p16(part)), cols]: every part of a head padded on its own."""
    a = a.reshape(heads, sum(parts), a.shape[1])
    out, at, to = np.zeros((heads, sum(p16(n) for n in parts), cols), a.dtype), 0, 0
    for n in parts:
        out[:, to:to + n, :a.shape[2]] = a[:, at:at + n]
        at, to = at + n, to + p16(n)
    return out.reshape(-1, cols)


def _head_transposed(a: np.ndarray, heads: int, dim: int) -> np.ndarray:
    """[heads * dim, K] -> [heads * p16(K), p64(dim)], each head's block transposed."""
    k = a.shape[1]
    out = np.zeros((heads, p16(k), p64(dim)), a.dtype)
    out[:, :k, :dim] = a.reshape(heads, dim, k).transpose(0, 2, 1)
    return out.reshape(-1, p64(dim))


class Goselix(DecoderModel):
    def __init__(self, runtime: B200Runtime, config: GoselixConfig, tensors, max_seq_len: int = 1024, batch: int = 1, precision: str = "bf16",
                 max_rows: int = 0, max_portion: int = 0):
        super().__init__(runtime, config, tensors, max_seq_len, batch, precision)
        wp, width = p64(config.width), config.width
        get, weight, vector = self._get, self._weight, self._vector

        descs = (L.LayerDesc * len(config.layers))()
        for i, (lc, d) in enumerate(zip(config.layers, descs)):
            pre, mx = f"l{i}.", lc.mixer
            mix = pre + "mix."
            d.parallel, d.norm1_w = 1, self._gains(pre + "norm1", width, wp)
            H, D, E = mx.heads, mx.dim, mx.vdim
            d.heads, d.dim, d.vdim = H, D, E
            if isinstance(mx, LatentConfig):
                P, Q, K = mx.rot_dim, mx.q_rank, mx.kv_rank
                d.mixer, d.rot_dims, d.q_rank, d.kv_rank, d.scale = L.MIX_LATENT, P, Q, K, mx.scale
                d.rot_freq = vector(rope_frequencies(P, mx.rot_base)) if P else None
                d.q_norm, d.kv_norm = self._gains(mix + "dq.norm", Q, p64(Q)), self._gains(mix + "dkv.norm", K, p16(K))
                down = get(mix + "dkv", K + P, width)
                fused = np.concatenate([_pad(get(mix + "dq", Q, width), p64(Q), wp), _pad(down[:K], p16(K), wp), _pad(down[K:], p16(P), wp)], axis=0)
                d.in_w = weight(mix + "in", _pad(fused, p64(fused.shape[0]), wp))
                d.uq_w = weight(mix + "uq", _head_parts(get(mix + "uq", H * (D + P), Q), H, (D, P), p64(Q)))
                uk, uv = get(mix + "uk", H * D, K), get(mix + "uv", H * E, K)
                d.uk_w = weight(mix + "uk", _head_transposed(uk, H, D))
                d.kv_w = weight(mix + "kv", np.concatenate([_head_rows(uk, H, D, p64(K)), _head_rows(uv, H, E, p64(K))], axis=0))
            else:
                d.mixer, d.rot_dims = L.MIX_RETENTION, mx.rot_dims
                d.rot_freq = vector(rope_frequencies(mx.rot_dims, mx.rot_base)) if mx.rot_dims else None
                d.powers = vector(np.asarray(mx.decay, np.float64)[:, None] ** np.arange(CHUNK + 1))
                rows = [_head_rows(get(mix + c, H * n, width), H, n, wp) for c, n in (("q", D), ("k", D), ("v", E), ("g", E))]
                fused = np.concatenate(rows, axis=0)
                d.in_w = weight(mix + "in", _pad(fused, p64(fused.shape[0]), wp))
            out = [_head_cols(get(mix + "o", width, H * E), H, E, wp)]
            if lc.mlp is not None:
                ff, fp, mlp = lc.mlp.ff, p64(lc.mlp.ff), pre + "mlp."
                d.norm2_w, d.ff_act = self._gains(pre + "norm2", width, wp), L.ACT_SILU_GLU
                if isinstance(lc.mlp, DenseConfig):
                    d.ff_in = weight(mlp + "in", self._glu_pairs(mlp + "gate", mlp + "up", ff, width))
                    out.append(_pad(get(mlp + "down", width, ff), wp, fp))
                else:
                    n = lc.mlp.experts
                    d.experts, d.top = n, lc.mlp.top
                    d.router = weight(mlp + "router", _pad(get(mlp + "router", n, width), p64(n), wp))
                    d.ff_in = weight(mlp + "in", np.concatenate([self._glu_pairs(f"{mlp}e{e}.gate", f"{mlp}e{e}.up", ff, width) for e in range(n)], axis=0))
                    d.ff_out = weight(mlp + "down", np.concatenate([_pad(get(f"{mlp}e{e}.down", width, ff), wp, fp) for e in range(n)], axis=0))
            d.out_w = weight(mix + "o", np.concatenate(out, axis=1))

        def fill(desc):
            desc.final_norm = self._gains("final.norm", width, wp)
            if config.loop:
                desc.loop_start, desc.loop_stop, desc.loop_times = config.loop
                step = np.zeros((config.loop[2], wp), np.float32)
                step[:, :width] = bf16_to_f32(get("loop.step", config.loop[2], width))
                desc.loop_step = vector(step)

        self._create(descs, max_rows, max_portion, fill)


def load(path: str, runtime: Optional[B200Runtime] = None, **kw) -> Goselix:
    """A model from a folder with ``config.json`` and ``model.safetensors``."""
    return load_folder(path, parse_config, Goselix, runtime, **kw)
