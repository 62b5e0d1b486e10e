"""Reader of .safetensors files: an 8-byte little-endian header length, a JSON header
(name -> dtype, shape, data_offsets) and the tensor bytes, memory-mapped."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

# BF16 has no numpy type: its bit patterns are returned as uint16
_DTYPES = {"F32": np.float32, "F16": np.float16, "BF16": np.uint16, "F64": np.float64, "I64": np.int64, "I32": np.int32,
           "I16": np.int16, "I8": np.int8, "U8": np.uint8, "BOOL": np.bool_}


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (np.asarray(bits, np.uint32) << np.uint32(16)).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    """Bit patterns (uint16) of finite fp32 values rounded to the nearest bf16, ties to even."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint16).reshape(np.shape(x))


class SafeTensors:
    def __init__(self, path: str):
        size = os.path.getsize(path)
        with open(path, "rb") as f:
            head = f.read(8)
            if len(head) != 8:
                raise ValueError(f"{path}: not a safetensors file")
            (n,) = struct.unpack("<Q", head)
            if n > size - 8:
                raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
            self._index = json.loads(f.read(n))
        self._index.pop("__metadata__", None)
        self._data = np.memmap(path, np.uint8, "r", offset=8 + n, shape=(size - 8 - n,)) if size > 8 + n else np.zeros(0, np.uint8)
        for name, t in self._index.items():
            a, b = t["data_offsets"]
            want = int(np.prod(t["shape"], dtype=np.int64)) * np.dtype(_DTYPES[t["dtype"]]).itemsize if t["dtype"] in _DTYPES else -1
            if a < 0 or b > self._data.size or b - a != want:
                raise ValueError(f"{path}: tensor {name} ({t['dtype']} {t['shape']}) does not fit its bytes [{a}, {b})")

    def __contains__(self, name: str) -> bool:
        return name in self._index

    def names(self):
        return list(self._index)

    def dtype(self, name: str) -> str:
        return self._index[name]["dtype"]

    def raw(self, name: str) -> np.ndarray:
        """The tensor as stored; BF16 as uint16 bit patterns."""
        if name not in self._index:
            raise KeyError(f"tensor {name} is missing")
        t = self._index[name]
        a, b = t["data_offsets"]
        return self._data[a:b].view(_DTYPES[t["dtype"]]).reshape(t["shape"])

    def bf16(self, name: str) -> np.ndarray:
        """Bit patterns (uint16) of a BF16 tensor."""
        a = self.raw(name)
        if self.dtype(name) != "BF16":
            raise ValueError(f"tensor {name} is {self.dtype(name)}, expected BF16")
        return np.asarray(a)

    def f32(self, name: str) -> np.ndarray:
        a = self.raw(name)
        return bf16_to_f32(a) if self.dtype(name) == "BF16" else np.asarray(a, np.float32)


def save(path: str, tensors: dict) -> None:
    """Writes ``{name: array}``; uint16 arrays are stored as BF16 bit patterns."""
    names = {np.dtype(v): k for k, v in _DTYPES.items()}
    index, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        b = np.ascontiguousarray(a).tobytes()
        index[name] = {"dtype": names[a.dtype], "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    head = json.dumps(index).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for b in blobs:
            f.write(b)
