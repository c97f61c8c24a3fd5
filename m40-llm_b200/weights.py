"""Reads a safetensors file: an 8-byte little-endian header length, the JSON header
(name -> dtype, shape, data_offsets), then the data. Tensors are views of the mapped file."""
from __future__ import annotations

import json
import mmap
import os
import struct

import numpy as np

_DTYPES = {"BF16": ("<u2", 2), "F16": ("<f2", 2), "F32": ("<f4", 4), "I32": ("<i4", 4)}


class TensorFile:
    def __init__(self, path: str):
        self._f = open(path, "rb")
        size = os.fstat(self._f.fileno()).st_size
        self._map = mmap.mmap(self._f.fileno(), 0, access=mmap.ACCESS_READ)
        if size < 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", self._map[:8])[0]
        if 8 + n > size:
            raise ValueError(f"{path}: header length {n} exceeds the file")
        self._base = 8 + n
        self.entries = {k: v for k, v in json.loads(self._map[8:8 + n]).items() if k != "__metadata__"}
        for name, e in self.entries.items():
            lo, hi = e["data_offsets"]
            width = _DTYPES.get(e["dtype"], (None, 0))[1]
            if not width or lo > hi or self._base + hi > size or hi - lo != width * int(np.prod(e["shape"], dtype=np.int64)):
                raise ValueError(f"{path}: bad entry {name}: {e}")

    def __contains__(self, name: str) -> bool:
        return name in self.entries

    def shape(self, name: str) -> tuple[int, ...]:
        return tuple(self.entries[name]["shape"])

    def raw(self, name: str) -> tuple[np.ndarray, str]:
        """(array, dtype name); bfloat16 comes as its uint16 bits."""
        if name not in self.entries:
            raise KeyError(f"tensor {name!r} is missing from the weights")
        e = self.entries[name]
        lo, hi = e["data_offsets"]
        np_type, width = _DTYPES[e["dtype"]]
        a = np.frombuffer(self._map, np_type, (hi - lo) // width, self._base + lo)
        return a.reshape(e["shape"]), e["dtype"]

    def f32(self, name: str) -> np.ndarray:
        a, dtype = self.raw(name)
        return bf16_to_f32(a) if dtype == "BF16" else a.astype(np.float32)

    def bf16(self, name: str) -> np.ndarray:
        """The tensor as bfloat16 bits (rounded to nearest even when the file holds wider values)."""
        a, dtype = self.raw(name)
        return a if dtype == "BF16" else f32_to_bf16(a.astype(np.float32))


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    x = np.asarray(x, np.float32)
    u = np.ascontiguousarray(x).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16).reshape(x.shape)


def write(path: str, tensors: dict[str, np.ndarray]):
    """Writes float arrays as BF16 and int32 arrays as I32 (for tests, benchmarks and converters)."""
    header, blobs, at = {}, [], 0
    for name, a in tensors.items():
        a = np.asarray(a)
        raw, dtype = (a.astype("<i4").tobytes(), "I32") if a.dtype.kind == "i" else (f32_to_bf16(a).tobytes(), "BF16")
        header[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for b in blobs:
            f.write(b)
