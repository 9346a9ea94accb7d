"""Rotary position tables, computed on the host in double and narrowed to f32.

Two layouts: `rope_tables` for the rotate-half rotation (both halves of a row equal), `pair_tables` for the interleaved one
(one column per pair), whose frequencies may be stretched for contexts beyond the trained one.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import numpy as np


def rope_tables(theta: float, head_dim: int, positions: int):
    """HfDecoderGraph.ropeTables (:436-462): computed in double, narrowed to f32, both halves equal."""
    half = head_dim // 2
    inv = np.power(float(theta), -2.0 * np.arange(half, dtype=np.float64) / head_dim)
    ang = np.arange(positions, dtype=np.float64)[:, None] * inv[None, :]
    cos = np.concatenate([np.cos(ang), np.cos(ang)], axis=1).astype(np.float32)
    sin = np.concatenate([np.sin(ang), np.sin(ang)], axis=1).astype(np.float32)
    return cos, sin


@dataclass(frozen=True)
class YarnScaling:
    """Frequencies interpolated by parts (YaRN): pairs that turn more than `fast` times over the `original` context keep their
    frequency, those that turn fewer than `slow` times have it divided by `factor`, with a linear ramp over the pairs between."""

    factor: float
    original: float
    fast: float
    slow: float

    @property
    def magnitude(self) -> float:
        """What cosine and sine are multiplied by."""
        return 0.1 * math.log(self.factor) + 1.0

    def apply(self, freqs: np.ndarray, dims: int, base: float) -> np.ndarray:
        def pair_of(turns: float) -> float:  # the (fractional) dimension whose pair makes that many turns
            return dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(pair_of(self.fast)), 0)
        hi = min(math.ceil(pair_of(self.slow)), dims - 1)
        ramp = np.clip((np.arange(freqs.shape[0], dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return freqs / self.factor * ramp + freqs * (1.0 - ramp)


@dataclass(frozen=True)
class Rotation:
    """Interleaved rotation of the first `dims` dimensions of a vector: pair i turns by position * base^(-2i / dims)."""

    dims: int
    base: float
    scaling: YarnScaling | None = None

    def __post_init__(self):
        if self.dims < 0 or self.dims % 2:
            raise ValueError(f"rotation over {self.dims} dimensions: an even number is needed")


def pair_tables(rot: Rotation, positions: int):
    """(cos, sin), f32 [positions, dims / 2], the scaling's magnitude multiplied in."""
    pairs = rot.dims // 2
    freqs = np.power(float(rot.base), -2.0 * np.arange(pairs, dtype=np.float64) / max(rot.dims, 1))
    magnitude = 1.0
    if rot.scaling is not None:
        freqs, magnitude = rot.scaling.apply(freqs, rot.dims, float(rot.base)), rot.scaling.magnitude
    ang = np.arange(positions, dtype=np.float64)[:, None] * freqs[None, :]
    return (np.cos(ang) * magnitude).astype(np.float32), (np.sin(ang) * magnitude).astype(np.float32)
