"""Rotary position encoding: the table of inverse frequencies.

inv_freq[i] = theta^(-2i / rotary_dim) in float32
(crates/model/src/components/positional/rope.rs:498-503 of the reference).  The
rotation itself runs inside the kernel that also norms the heads and writes the
cache; this part owns the constants and hands them over through `fused_rotary`.
"""
from __future__ import annotations

import math

import numpy as np
import torch

from .registry import POSITIONS
from .spec import RotarySpec, YarnScaling


def scaled_frequencies(rotary_dim: int, theta: float, scaling) -> np.ndarray:
    """theta^(-2i / rotary_dim) slowed down (`RotaryScaling`, `YarnScaling`), worked out in double precision and rounded once."""
    f = float(theta) ** (-2.0 * np.arange(rotary_dim // 2, dtype=np.float64) / rotary_dim)
    if isinstance(scaling, YarnScaling):
        at = lambda turns: rotary_dim * math.log(scaling.original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
        low, high = max(math.floor(at(scaling.fast)), 0), min(math.ceil(at(scaling.slow)), rotary_dim - 1)
        r = np.clip((np.arange(rotary_dim // 2, dtype=np.float64) - low) / max(high - low, 0.001), 0.0, 1.0)
        return (f / scaling.factor * r + f * (1.0 - r)).astype(np.float32)
    if scaling.original is None:
        return (f / scaling.factor).astype(np.float32)
    wave = 2.0 * np.pi / f
    s = (scaling.original / wave - scaling.low) / (scaling.high - scaling.low)
    ramp = (1.0 - s) * f / scaling.factor + s * f
    out = np.where(wave < scaling.original / scaling.high, f, np.where(wave > scaling.original / scaling.low, f / scaling.factor, ramp))
    return out.astype(np.float32)


def amplitude(scaling) -> float:
    """What sine and cosine are multiplied by under a scaling of the frequencies."""
    return 0.1 * math.log(scaling.factor) + 1.0 if isinstance(scaling, YarnScaling) else 1.0


def inverse_frequencies(rotary_dim: int, theta: float) -> np.ndarray:
    i = np.arange(rotary_dim // 2, dtype=np.float32)
    exponent = (np.float32(-2.0) * i / np.float32(rotary_dim)).astype(np.float32)
    return np.power(np.float32(theta), exponent).astype(np.float32)


@POSITIONS.register("rotary")
class RotaryTable:
    @staticmethod
    def declare(spec: RotarySpec) -> dict:
        return {}

    def __init__(self, spec: RotarySpec, weights: dict, ctx):
        if spec.dim % 2 or spec.dim > spec.head_dim or spec.dim <= 0:
            raise ValueError(f"rotary_dim {spec.dim} must be even and at most head_dim {spec.head_dim}")
        self.spec = spec
        table = inverse_frequencies(spec.dim, spec.theta) if spec.scaling is None else scaled_frequencies(spec.dim, spec.theta, spec.scaling)
        self.inv_freq = torch.from_numpy(table).to(ctx.device)
        self.amplitude = amplitude(spec.scaling)

    def fused_rotary(self):
        if self.amplitude != 1.0:
            raise NotImplementedError("this mixer's kernels turn by plain sines and cosines; a scaling with an amplitude "
                                      "needs a mixer that asks for scaled_rotary()")
        return self.inv_freq, self.spec.dim

    def scaled_rotary(self):
        """(inv_freq, rotated features, factor on sine and cosine)."""
        return self.inv_freq, self.spec.dim, self.amplitude
