"""What the layer-list decoders of this package have in common: the storage rules of
``caten_b200_decoder_create`` (include/caten_b200.h), uploads, and the step entry points.  A model lays its
weights out in ``caten_b200_layer_desc`` / ``caten_b200_decoder_desc`` and calls :meth:`DecoderModel._create`."""
from __future__ import annotations

import ctypes as C
import json
import math
import os
from typing import Callable, Optional, Sequence

import numpy as np

from . import _lib as L
from .model import Model
from .runtime import B200Buffer, B200Runtime
from .safetensors import SafeTensors, bf16_to_f32
from .synthetic import Packed


def p16(n: int) -> int:
    return -(-n // 16) * 16


def p64(n: int) -> int:
    return -(-n // 64) * 64


def p128(n: int) -> int:
    return -(-n // 128) * 128


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


class DecoderModel(Model):
    def __init__(self, runtime: B200Runtime, config, tensors, max_seq_len: int, batch: int, precision):
        """``tensors``: name -> bf16 bit patterns (uint16), e.g. ``SafeTensors.bf16`` behind a mapping."""
        self.rt, self.config, self.batch, self.max_seq_len, self.vocab_size = runtime, config, batch, max_seq_len, config.vocab
        self.precision = L.PRECISIONS[precision] if isinstance(precision, str) else int(precision)
        self._tensors, self._bufs, self._weights, self.weights = tensors, [], [], {}
        self._h = None

    def _get(self, name, *shape):
        a = self._tensors[name]
        if tuple(a.shape) != shape:
            raise ValueError(f"tensor {name} is {tuple(a.shape)}, expected {shape}")
        return a

    def _weight(self, name, a):
        a = np.ascontiguousarray(a, dtype=np.uint16)
        w = self.rt.upload_weight(Packed(L.BF16, a.shape[0], a.shape[1], a.view(np.uint8).reshape(-1)))
        self._weights.append(w)
        self.weights[name] = w
        return w.handle

    def _vector(self, a):
        b = self.rt.transfer_from_array(np.ascontiguousarray(a, dtype=np.float32))
        self._bufs.append(b)
        return b.ptr

    def _gains(self, name, n, padded):
        """[n] bf16 -> device fp32, padded with zeros."""
        v = np.zeros(padded, np.float32)
        v[:n] = bf16_to_f32(self._get(name, n))
        return self._vector(v)

    def _scalar(self, name):
        return float(bf16_to_f32(self._get(name)).reshape(()))

    def _glu_pairs(self, gate, up, ff, width):
        """Rows of gate and up in turn, [2 * p64(ff), p64(width)]."""
        pair = np.zeros((p64(ff), 2, p64(width)), np.uint16)
        pair[:ff, 0, :width] = self._get(gate, ff, width)
        pair[:ff, 1, :width] = self._get(up, ff, width)
        return pair.reshape(2 * p64(ff), p64(width))

    def _create(self, descs, max_rows: int, max_portion: int, fill: Callable) -> None:
        """``fill(desc)`` sets what differs between designs (eps, norm before the head, loop)."""
        cfg, wp = self.config, p64(self.config.width)
        desc = L.DecoderDesc()
        desc.n_layers, desc.width, desc.vocab, desc.max_seq_len, desc.batch = len(cfg.layers), cfg.width, cfg.vocab, self.max_seq_len, self.batch
        desc.precision, desc.max_rows, desc.max_portion, desc.eps = self.precision, max_rows, max_portion, cfg.eps
        desc.embed = self._weight("embed", _pad(self._get("embed", cfg.vocab, cfg.width), cfg.vocab, wp))
        desc.head = self._weight("head", _pad(self._get("head", cfg.vocab, cfg.width), cfg.vocab, wp))
        fill(desc)
        desc.layers = descs
        h = C.c_void_p()
        L.check(self.rt.ctx, self.rt.lib.caten_b200_decoder_create(self.rt.ctx, C.byref(desc), C.byref(h)))
        self._h = h
        self._tensors = None
        self.linear_weight_bytes = sum(w.packed_nbytes for w in self._weights)
        self._dev_ids = self.rt.open_buffer((2, self.batch), np.int64)  # ping-pong ids for device-resident decode

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


def load_folder(path: str, parse_config: Callable, model: Callable, runtime: Optional[B200Runtime] = None, **kw):
    """A model from a folder with ``config.json`` and ``model.safetensors``."""
    with open(os.path.join(path, "config.json")) as f:
        config = parse_config(json.load(f))
    return model(runtime or B200Runtime(0), config, _Bf16Tensors(SafeTensors(os.path.join(path, "model.safetensors"))), **kw)
