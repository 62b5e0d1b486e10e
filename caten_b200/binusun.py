"""Binusun: a decoder whose layers alternate between gated sliding-window attention (grouped query
heads, rotary positions, normalised q and k) and RWKV-style time mixing, with RMS norms of one scalar
gain before and after every sublayer and a range of layers that runs several times with the same
weights, each pass fed a projection of the stream and the embedding output.

``load`` reads a folder with ``config.json`` and ``model.safetensors``; :class:`Binusun` lays the
weights out the way ``caten_b200_decoder_create`` takes them (include/caten_b200.h) and steps the model
through it.  Every size and constant comes from the configuration.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import numpy as np

from . import _lib as L
from .decoder import DecoderModel, _head_cols, _head_rows, _head_vec, _pad, load_folder, p16, p64, p128, rope_frequencies
from .runtime import B200Runtime
from .safetensors import bf16_to_f32

ARCHITECTURE = "Binusun"


# ---- configuration ------------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    rot_dims: int
    rot_base: float
    rot_scaling: Optional[Tuple[float, float, float, float]]   # factor, low, high, original
    scale: float


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: object           # AttentionConfig or WkvConfig
    ff: Optional[int]       # width of the gated feed-forward, None: no feed-forward


@dataclass(frozen=True)
class BinusunConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: Tuple[LayerConfig, ...]
    loop: Optional[Tuple[int, int, int]]   # start, stop, times


def _attention(m: dict) -> AttentionConfig:
    rot, sc = m["rot"], m["rot"].get("scaling")
    return AttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["mask"]["size"]), int(rot["dims"]), float(rot["base"]),
                           tuple(float(sc[k]) for k in ("factor", "low", "high", "original")) if sc else None, float(m["scale"]))


def _wkv(m: dict) -> WkvConfig:
    return WkvConfig(int(m["heads"]), int(m["dim"]))


_MIXERS = {"attention": _attention, "wkv": _wkv}


def parse_config(cfg: dict) -> BinusunConfig:
    if cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCHITECTURE}")
    layers = []
    for i, l in enumerate(cfg["layers"]):
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
        mlp = l.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(LayerConfig(_MIXERS[l["type"]](l["mixer"]), int(mlp["ff"]) if mlp is not None else None))
    loop = cfg.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
    return BinusunConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]), float(cfg["logit_scale"]), tuple(layers), loop or None)


class Binusun(DecoderModel):
    def __init__(self, runtime: B200Runtime, config: BinusunConfig, tensors, max_seq_len: int = 1024, batch: int = 1, precision: str = "bf16",
                 max_rows: int = 0, max_portion: int = 0):
        """``tensors``: name -> bf16 bit patterns (uint16), e.g. ``SafeTensors.bf16`` behind a mapping."""
        super().__init__(runtime, config, tensors, max_seq_len, batch, precision)
        wp, width = p64(config.width), config.width
        get, weight, vector, scalar = self._get, self._weight, self._vector, self._scalar
        descs = (L.LayerDesc * len(config.layers))()
        for i, (lc, d) in enumerate(zip(config.layers, descs)):
            pre, mx = f"l{i}.", lc.mixer
            mix = pre + "mix."
            d.norm1, d.norm1b = scalar(pre + "norm1"), scalar(pre + "norm1b")
            if isinstance(mx, AttentionConfig):
                H, G, D, E = mx.heads, mx.kv_heads, mx.dim, mx.vdim
                d.mixer, d.heads, d.dim, d.kv_heads, d.vdim, d.window = L.MIX_ATTENTION, H, D, G, E, mx.window
                if mx.window < 1 or H % G:
                    raise ValueError(f"layer {i}: window {mx.window}, heads {H} / {G}")
                d.rot_dims, d.qk_norm, d.gated, d.scale = mx.rot_dims, 1, 1, mx.scale
                d.rot_freq = vector(rope_frequencies(mx.rot_dims, mx.rot_base, mx.rot_scaling)) if mx.rot_dims else None
                rows = [_head_rows(get(mix + "q", H * D, width), H, D, wp), _head_rows(get(mix + "k", G * D, width), G, D, wp),
                        _head_rows(get(mix + "v", G * E, width), G, E, wp), _pad(get(mix + "g", H, width), H, wp)]
                fused = np.concatenate(rows, axis=0)
                d.in_w = weight(mix + "in", _pad(fused, p64(fused.shape[0]), wp))
                d.out_w = weight(mix + "o", _head_cols(get(mix + "o", width, H * E), H, E, wp))
            else:
                H, D = mx.heads, mx.dim
                d.mixer, d.heads, d.dim = L.MIX_WKV, H, D
                w1 = tensors[mix + "w1"]
                rank = w1.shape[0]
                gr, low = p128(H * p16(D)), p64(rank)
                if low > gr:
                    gr = p128(low)
                d.group_rows, d.low_rank = gr, low
                groups = [_pad(_head_rows(get(mix + c, H * D, width), H, D, wp), gr, wp) for c in "rkvg"]
                d.in_w = weight(mix + "in", np.concatenate(groups + [_pad(get(mix + "w1", rank, width), low, wp)], axis=0))
                d.w2 = weight(mix + "w2", _pad(_head_rows(get(mix + "w2", H * D, rank), H, D, low), p64(H * p16(D)), low))
                mu = np.zeros((5, wp), np.float32)
                for j, c in enumerate("rkvgw"):
                    mu[j, :width] = bf16_to_f32(get(f"{mix}mu.{c}", width))
                d.mu = vector(mu)
                d.w0 = vector(_head_vec(bf16_to_f32(get(mix + "w0", H * D)), H, D))
                d.u = vector(_head_vec(bf16_to_f32(get(mix + "u", H, D)), H, D))
                d.norm = vector(_head_vec(bf16_to_f32(get(mix + "norm", H * D)), H, D))
                d.out_w = weight(mix + "o", _head_cols(get(mix + "o", width, H * D), H, D, wp))
            if lc.ff is not None:
                ff, fp = lc.ff, p64(lc.ff)
                d.norm2, d.norm2b = scalar(pre + "norm2"), scalar(pre + "norm2b")
                d.ff_in = weight(pre + "mlp.in", self._glu_pairs(pre + "mlp.gate", pre + "mlp.up", ff, width))
                d.ff_out = weight(pre + "mlp.down", _pad(get(pre + "mlp.down", width, ff), wp, fp))

        def fill(desc):
            desc.final_gain = scalar("final.norm") * config.logit_scale
            if config.loop:
                desc.loop_start, desc.loop_stop, desc.loop_times = config.loop
                w = get("loop.in", width, 2 * width)
                desc.loop_in = weight("loop.in", np.concatenate([_pad(w[:, :width], wp, wp), _pad(w[:, width:], wp, wp)], axis=1))

        self._create(descs, max_rows, max_portion, fill)


def load(path: str, runtime: Optional[B200Runtime] = None, **kw) -> Binusun:
    """A model from a folder with ``config.json`` and ``model.safetensors``."""
    return load_folder(path, parse_config, Binusun, runtime, **kw)
