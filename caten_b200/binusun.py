"""Binusun: a decoder whose layers alternate between gated sliding-window attention (grouped query
heads, rotary positions, normalised q and k) and RWKV-style time mixing, with RMS norms of one scalar
gain before and after every sublayer and a range of layers that runs several times with the same
weights, each pass fed a projection of the stream and the embedding output.

``load`` reads a folder with ``config.json`` and ``model.safetensors``; :class:`Binusun` lays the
weights out the way ``caten_b200_decoder_create`` takes them (include/caten_b200.h) and steps the model
through it.  Every size and constant comes from the configuration.
"""
from __future__ import annotations

import ctypes as C
import json
import math
import os
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import numpy as np

from . import _lib as L
from .model import Model
from .runtime import B200Buffer, B200Runtime
from .safetensors import SafeTensors, bf16_to_f32
from .synthetic import Packed

ARCHITECTURE = "Binusun"


def p16(n: int) -> int:
    return -(-n // 16) * 16


def p64(n: int) -> int:
    return -(-n // 64) * 64


def p128(n: int) -> int:
    return -(-n // 128) * 128


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


def rope_frequencies(dims: int, base: float, scaling: Optional[Sequence[float]] = None) -> np.ndarray:
    """Angle per position of pair i = base^(-2i/dims).  With ``scaling`` (factor, low, high, original) as in
    Llama 3.1: kept for wavelengths below original / high, divided by factor above original / low, and
    interpolated in between."""
    f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims) if dims else np.zeros(0)
    if scaling is not None and dims:
        factor, low, high, original = scaling
        wl = 2.0 * math.pi / f
        with np.errstate(divide="ignore", invalid="ignore"):
            s = (original / wl - low) / (high - low)
        mid = (1.0 - s) * f / factor + s * f
        f = np.where(wl < original / high, f, np.where(wl > original / low, f / factor, mid))
    return f


# ---- weight layout (bf16 bit patterns, padded with zeros) ------------------------------------------
def _pad(a: np.ndarray, rows: int, cols: int) -> np.ndarray:
    out = np.zeros((rows, cols), a.dtype)
    out[:a.shape[0], :a.shape[1]] = a
    return out


def _head_rows(a: np.ndarray, heads: int, dim: int, cols: int) -> np.ndarray:
    """[heads * dim, K] -> [heads * p16(dim), cols]."""
    out = np.zeros((heads, p16(dim), cols), a.dtype)
    out[:, :dim, :a.shape[1]] = a.reshape(heads, dim, a.shape[1])
    return out.reshape(heads * p16(dim), cols)


def _head_cols(a: np.ndarray, heads: int, dim: int, rows: int) -> np.ndarray:
    """[N, heads * dim] -> [rows, p64(heads * p16(dim))]."""
    out = np.zeros((rows, heads, p16(dim)), a.dtype)
    out[:a.shape[0], :, :dim] = a.reshape(a.shape[0], heads, dim)
    return _pad(out.reshape(rows, -1), rows, p64(heads * p16(dim)))


def _head_vec(a: np.ndarray, heads: int, dim: int) -> np.ndarray:
    """[heads * dim] fp32 -> [p64(heads * p16(dim))]."""
    out = np.zeros(p64(heads * p16(dim)), np.float32)
    out[:heads * p16(dim)].reshape(heads, p16(dim))[:, :dim] = a.reshape(heads, dim)
    return out


class Binusun(Model):
    def __init__(self, runtime: B200Runtime, config: BinusunConfig, tensors, max_seq_len: int = 1024, batch: int = 1, precision: str = "bf16",
                 max_rows: int = 0, max_portion: int = 0):
        """``tensors``: name -> bf16 bit patterns (uint16), e.g. ``SafeTensors.bf16`` behind a mapping."""
        self.rt, self.config, self.batch, self.max_seq_len, self.vocab_size = runtime, config, batch, max_seq_len, config.vocab
        self.precision = L.PRECISIONS[precision] if isinstance(precision, str) else int(precision)
        self._bufs, self._weights, self.weights = [], [], {}
        self._h = None
        wp, width = p64(config.width), config.width

        def get(name, *shape):
            a = tensors[name]
            if tuple(a.shape) != shape:
                raise ValueError(f"tensor {name} is {tuple(a.shape)}, expected {shape}")
            return a

        def weight(name, a):
            a = np.ascontiguousarray(a, dtype=np.uint16)
            w = runtime.upload_weight(Packed(L.BF16, a.shape[0], a.shape[1], a.view(np.uint8).reshape(-1)))
            self._weights.append(w)
            self.weights[name] = w
            return w.handle

        def vector(a):
            b = runtime.transfer_from_array(np.ascontiguousarray(a, dtype=np.float32))
            self._bufs.append(b)
            return b.ptr

        def scalar(name):
            return float(bf16_to_f32(get(name)).reshape(()))

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
                pair = np.zeros((fp, 2, wp), np.uint16)
                pair[:ff, 0, :width] = get(pre + "mlp.gate", ff, width)
                pair[:ff, 1, :width] = get(pre + "mlp.up", ff, width)
                d.ff_in = weight(pre + "mlp.in", pair.reshape(2 * fp, wp))
                d.ff_out = weight(pre + "mlp.down", _pad(get(pre + "mlp.down", width, ff), wp, fp))
        desc = L.DecoderDesc()
        desc.n_layers, desc.width, desc.vocab, desc.max_seq_len, desc.batch = len(config.layers), width, config.vocab, max_seq_len, batch
        desc.precision, desc.max_rows, desc.max_portion = self.precision, max_rows, max_portion
        desc.eps, desc.final_gain = config.eps, scalar("final.norm") * config.logit_scale
        desc.embed = weight("embed", _pad(get("embed", config.vocab, width), config.vocab, wp))
        desc.head = weight("head", _pad(get("head", config.vocab, width), config.vocab, wp))
        if config.loop:
            desc.loop_start, desc.loop_stop, desc.loop_times = config.loop
            w = get("loop.in", width, 2 * width)
            desc.loop_in = weight("loop.in", np.concatenate([_pad(w[:, :width], wp, wp), _pad(w[:, width:], wp, wp)], axis=1))
        desc.layers = descs
        h = C.c_void_p()
        L.check(runtime.ctx, runtime.lib.caten_b200_decoder_create(runtime.ctx, C.byref(desc), C.byref(h)))
        self._h = h
        self.linear_weight_bytes = sum(w.packed_nbytes for w in self._weights)
        self._dev_ids = runtime.open_buffer((2, batch), np.int64)  # ping-pong ids for device-resident decode

    # -- steps --
    def step(self, tokens, n: int, want=(), ids: bool = False):
        """The next tokens [batch, s] of every sequence at positions n .. (0 starts new sequences, otherwise
        where the previous step ended).  Returns (logits [batch, len(want), vocab] at the places ``want`` of
        this step, argmax ids [batch] or None)."""
        tok = np.ascontiguousarray(tokens, dtype=np.int64).reshape(self.batch, -1)
        want = np.asarray(want, np.int64).reshape(-1)
        places, back = np.unique(want, return_inverse=True)
        places = np.ascontiguousarray(places)
        lg = np.empty((self.batch, places.size, self.vocab_size), np.float32)
        out = np.empty(self.batch, np.int64) if ids else None
        L.check(self.rt.ctx, self.rt.lib.caten_b200_decoder_step(self._h, tok.ctypes.data, tok.shape[1], int(n), places.ctypes.data if places.size else None,
                                                                 places.size, lg.ctypes.data if places.size else None,
                                                                 out.ctypes.data if ids else None))
        return lg[:, back], out

    def layer_outputs(self, tokens, n: int = 0) -> np.ndarray:
        """Residual stream after every layer run of one step, [runs, batch * s, width] (for checks)."""
        tok = np.ascontiguousarray(tokens, dtype=np.int64).reshape(self.batch, -1)
        buf = np.zeros((int(self.rt.lib.caten_b200_decoder_runs(self._h)), tok.size, self.config.width), np.float32)
        L.check(self.rt.ctx, self.rt.lib.caten_b200_decoder_capture(self._h, buf.ctypes.data))
        try:
            self.step(tok, n)
            self.rt.sync()
        finally:
            self.rt.lib.caten_b200_decoder_capture(self._h, None)
        return buf

    def _step(self, tokens: np.ndarray, n: int) -> np.ndarray:
        return self.step(tokens, n, ids=True)[1]

    def _step_device(self, ids: B200Buffer, s: int, n: int, out: Optional[B200Buffer]) -> None:
        if ids.dtype != np.int64:
            raise ValueError("ids must be int64")
        L.check(self.rt.ctx, self.rt.lib.caten_b200_decoder_step_device(self._h, ids.ptr, s, n, out.ptr if out is not None else None))

    def _decode(self, first_ids: B200Buffer, n: int, steps: int, out: Optional[B200Buffer]) -> None:
        L.check(self.rt.ctx, self.rt.lib.caten_b200_decoder_decode(self._h, first_ids.ptr, n, steps, out.ptr if out is not None else None))

    def _logits_ptr(self) -> int:
        return self.rt.lib.caten_b200_decoder_logits(self._h)

    @property
    def cache_nbytes(self) -> int:
        """Device memory held by the attention rings and the recurrent states."""
        return int(self.rt.lib.caten_b200_decoder_cache_nbytes(self._h))

    @property
    def launch_count(self) -> int:
        return int(self.rt.lib.caten_b200_decoder_launch_count(self._h))

    def close(self):
        if getattr(self, "_h", None):
            if self.rt.ctx is None:   # the runtime (and with it the stream the model uses) is already gone
                self._h = None
                return
            self.rt.lib.caten_b200_decoder_destroy(self._h)
            self._h = None
            for w in self._weights:
                w.close()
            for b in self._bufs:
                b.close()
            self._dev_ids.close()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


class _Bf16Tensors:
    def __init__(self, st: SafeTensors):
        self._st = st

    def __getitem__(self, name):
        return self._st.bf16(name)


def load(path: str, runtime: Optional[B200Runtime] = None, **kw) -> Binusun:
    """A model from a folder with ``config.json`` and ``model.safetensors``."""
    with open(os.path.join(path, "config.json")) as f:
        config = parse_config(json.load(f))
    return Binusun(runtime or B200Runtime(0), config, _Bf16Tensors(SafeTensors(os.path.join(path, "model.safetensors"))), **kw)
