"""Rotary position encoding as a part, and the frequencies of rotations that mixers apply themselves."""
from __future__ import annotations

import math

import numpy as np
import torch

from .base import PositionEncoding, register_part


def rotation_frequencies(dims: int, base: float, scaling: dict | None = None) -> tuple[np.ndarray, float]:
    """Angle per position of each of the ``dims / 2`` pairs (worked out in 64-bit, rounded to 32-bit once: a kernel's angle is
    float(position) * frequency in 32-bit), and the amplitude that cosines and sines are multiplied by.

    Without ``scaling``: base^(-2i / dims) and 1.  ``scaling`` = {``factor``, ``original``, ``fast``, ``slow``} is YaRN's: a pair that turns at least ``fast``
    times over ``original`` positions keeps its frequency, one that turns at most ``slow`` times has it divided by ``factor``, those between
    (counted in pairs, the ends rounded outwards) blend linearly; the amplitude is 0.1 ln(factor) + 1."""
    index = np.arange(dims // 2, dtype=np.float64)
    frequency = np.power(float(base), -2.0 * index / float(max(dims, 1)))
    if scaling is None:
        return frequency.astype(np.float32), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    low = max(math.floor(pair_of(float(scaling["fast"]))), 0)
    high = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
    ramp = np.clip((index - low) / max(high - low, 0.001), 0.0, 1.0)
    return (frequency / factor * ramp + frequency * (1.0 - ramp)).astype(np.float32), 0.1 * math.log(factor) + 1.0


class RotaryEmbedding(PositionEncoding):
    """Half-split rotation of q and k (src/operators.cpp:47-78).

    params: ``rotary_dim`` (how many leading elements of a head rotate; the reference
    rotates the whole head), ``theta``.  The frequency of pair d is
    ``theta ** (-2 d / rotary_dim)`` evaluated in 32-bit, as the reference's ``std::pow``
    on floats does; the angle ``float(position) * frequency`` and its sine and cosine
    are 32-bit inside the kernel.  Keys are cached after rotation, so the cache never
    depends on this part.
    """

    capturable = True

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.rotary_dim = int(spec["rotary_dim"])
        self.theta = float(spec["theta"])
        half = self.rotary_dim // 2
        exponent = (np.float32(-2.0) * np.arange(half, dtype=np.float32)) / np.float32(self.rotary_dim)
        inv_freq = np.power(np.float32(self.theta), exponent, dtype=np.float32)
        self.inv_freq = torch.from_numpy(inv_freq).to(runtime.device)

    def rotary_table(self):
        return self.inv_freq, self.rotary_dim


class NoPositionEncoding(PositionEncoding):
    """Leaves q and k as they are (a mixer that needs no positions)."""

    capturable = True

    def rotary_table(self):
        return None

    def apply(self, qkv, ctx, q_heads, kv_heads, head_dim) -> None:
        return None


register_part("position", "rotary", RotaryEmbedding)
register_part("position", "none", NoPositionEncoding)
