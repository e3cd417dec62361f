"""Rotary position encoding: the table of inverse frequencies.

inv_freq[i] = theta^(-2i / rotary_dim) in float32
(crates/model/src/components/positional/rope.rs:498-503 of the reference).  The
rotation itself runs inside the kernel that also norms the heads and writes the
cache; this part owns the constants and hands them over through `fused_rotary`.
"""
from __future__ import annotations

import numpy as np
import torch

from .registry import POSITIONS
from .spec import RotarySpec


def scaled_frequencies(rotary_dim: int, theta: float, scaling) -> np.ndarray:
    """theta^(-2i / rotary_dim) slowed down (`RotaryScaling`), worked out in double precision and rounded once."""
    f = float(theta) ** (-2.0 * np.arange(rotary_dim // 2, dtype=np.float64) / rotary_dim)
    if scaling.original is None:
        return (f / scaling.factor).astype(np.float32)
    wave = 2.0 * np.pi / f
    s = (scaling.original / wave - scaling.low) / (scaling.high - scaling.low)
    ramp = (1.0 - s) * f / scaling.factor + s * f
    out = np.where(wave < scaling.original / scaling.high, f, np.where(wave > scaling.original / scaling.low, f / scaling.factor, ramp))
    return out.astype(np.float32)


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

    def fused_rotary(self):
        return self.inv_freq, self.spec.dim
