"""Builds a host.StackModel from named tensors: packs the projections that share an input into one matrix, uploads every
layer's weights once (a looped layer runs several times on the same weights, with its own cache per run) and makes the
rotation tables.
"""
from __future__ import annotations

import math

import numpy as np

from .. import native


def rotary_tables(base: float, dims: int, scaling: dict | None) -> tuple[np.ndarray, float]:
    """(turns per position of every pair, f64; amplitude). With `scaling` (factor, original, fast, slow) the frequencies
    follow YaRN: pairs that turn more than `fast` times within `original` positions keep their frequency, pairs that turn
    less than `slow` times are slowed down by `factor`, a linear ramp in between; the amplitude is 0.1 ln(factor) + 1."""
    pair = np.arange(dims // 2, dtype=np.float64)
    freq = float(base) ** (-2.0 * pair / dims)
    amp = 1.0
    if scaling:
        factor = float(scaling["factor"])

        def pair_with(turns):
            return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(pair_with(scaling["fast"])), 0)
        hi = min(math.ceil(pair_with(scaling["slow"])), dims - 1)
        ramp = np.clip((pair - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        freq = freq / factor * ramp + freq * (1.0 - ramp)
        amp = 0.1 * math.log(factor) + 1.0
    return freq / (2.0 * math.pi), amp


class StackWeights:
    """Device copies of one model's tensors, made on demand and kept by `nat`."""

    def __init__(self, nat, tensors):
        self.nat, self.t = nat, tensors
        self._mat: dict[tuple, int] = {}
        self._vec: dict[tuple, int] = {}

    def shape(self, name: str) -> tuple[int, ...]:
        return self.t.shape(name)

    def matrix(self, *names: str, shapes=None, rows: int = 0) -> int:
        """bf16 rows of the named [out, in] matrices, one after the other; zero rows follow up to `rows` of them."""
        if names not in self._mat:
            for n, shape in zip(names, shapes or ()):
                if self.t.shape(n) != tuple(shape):
                    raise ValueError(f"tensor {n}: shape {self.t.shape(n)}, expected {tuple(shape)}")
            parts = [self.t.bf16(n) for n in names]
            missing = rows - sum(len(p) for p in parts)
            if missing > 0:
                parts.append(np.zeros((missing, *parts[0].shape[1:]), np.uint16))
            self._mat[names] = self.nat.buf(np.concatenate(parts)).ptr
        return self._mat[names]

    def blocks_transposed(self, name: str, shape, blocks: int) -> int:
        """bf16 copy of a matrix [blocks * n][k] with every block of n rows transposed: [blocks * k][n]."""
        key = (name, "transposed", blocks)
        if key not in self._mat:
            if self.t.shape(name) != tuple(shape):
                raise ValueError(f"tensor {name}: shape {self.t.shape(name)}, expected {tuple(shape)}")
            a = self.t.bf16(name).reshape(blocks, shape[0] // blocks, shape[1])
            self._mat[key] = self.nat.buf(np.ascontiguousarray(a.transpose(0, 2, 1))).ptr
        return self._mat[key]

    def vectors(self, names, sizes, total: int) -> int:
        """f32 copies of several vectors, one after the other, zeros up to `total` values."""
        key = ("vectors", *names)
        if key not in self._vec:
            out, at = np.zeros(total, np.float32), 0
            for n, size in zip(names, sizes):
                a = self.t.f32(n).reshape(-1)
                if a.size != size:
                    raise ValueError(f"tensor {n}: {a.size} values, expected {size}")
                out[at:at + size] = a
                at += size
            self._vec[key] = self.nat.buf(out).ptr
        return self._vec[key]

    def vector(self, name: str, size: int, row: int | None = None) -> int:
        """f32 copy of a vector, or of one row of a matrix."""
        key = (name, row)
        if key not in self._vec:
            a = self.t.f32(name)
            a = (a if row is None else a[row]).reshape(-1)
            if a.size != size:
                raise ValueError(f"tensor {name}: {a.size} values, expected {size}")
            self._vec[key] = self.nat.buf(a).ptr
        return self._vec[key]

    def table(self, values: np.ndarray) -> int:
        key = ("table", values.tobytes())
        if key not in self._vec:
            self._vec[key] = self.nat.buf(np.ascontiguousarray(values, np.float64)).ptr
        return self._vec[key]

    def rms(self, name: str, size: int, eps: float, groups: int = 1) -> native.Norm:
        return native.Norm(native.NORM_RMS, eps, 0.0, self.vector(name, size), None, groups, 0)

    def dynamic_tanh(self, name: str, size: int) -> native.Norm:
        alpha = self.t.f32(name + ".alpha").reshape(-1)
        if alpha.size != 1:
            raise ValueError(f"tensor {name}.alpha: {alpha.size} values, expected one")
        return native.Norm(native.NORM_DYT, 0.0, float(alpha[0]), self.vector(name, size), self.vector(name + ".b", size))
