"""Rotate-half rotary position encoding.

inv_freq[i] = 1 / theta^(2i/Dh) for i < Dh/2, made in float32 exactly as the reference
does (src/ops/cpu_backend.cpp:14-21: ``1.f / pow(theta, float(2i)/float(Dh))`` with theta
a float32); the angle pos*inv_freq and its sine and cosine are float32 in the kernel.
The whole head is rotated; there is no scaling of positions.
"""
from __future__ import annotations

import math
from typing import Optional, Sequence, Tuple

import torch

from .base import PositionEncoding, register_position_encoding

Tensor = torch.Tensor


def rotary_frequencies(dims: int, base: float, factor: float = 1.0,
                       scaling: Optional[Sequence[float]] = None) -> Tensor:
    """base^(-2i/dims) / factor for i < dims/2, made in float64 and rounded to float32 once.  ``scaling`` = (factor, low,
    high, original): by how often a frequency's wavelength fits into ``original`` positions, n = original * f / (2 pi),
    it is divided by the factor (n < low), kept (n > high) or blended, (1 - s) f / factor + s f with
    s = (n - low) / (high - low)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / float(max(dims, 1))) / float(factor)
    if scaling is not None:
        by, low, high, original = (float(v) for v in scaling)
        n = original * f / (2.0 * math.pi)
        s = (n - low) / (high - low) if high != low else torch.zeros_like(n)
        f = torch.where(n > high, f, torch.where(n < low, f / by, (1.0 - s) * f / by + s * f))
    return f.to(torch.float32)


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float,
                     slow: float) -> Tuple[Tensor, float]:
    """(frequencies, factor on the sines and cosines) of YaRN scaling.  Pair i turns original * f_i / (2 pi) times within
    ``original`` positions; t(n) = dims * ln(original / (2 pi n)) / (2 ln base) is the (fractional) pair that turns n
    times.  Pairs up to lo = max(floor t(fast), 0) keep their frequency, those from hi = min(ceil t(slow), dims - 1) on
    are divided by the factor, between them the two are blended linearly in i; the sines and cosines are multiplied by
    0.1 ln(factor) + 1.  Made in float64 and rounded to float32 once."""
    def pair_turning(n: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * n)) / (2.0 * math.log(base))

    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / float(max(dims, 1)))
    lo, hi = max(math.floor(pair_turning(fast)), 0), min(math.ceil(pair_turning(slow)), dims - 1)
    r = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return (f / factor * r + f * (1.0 - r)).to(torch.float32), 0.1 * math.log(factor) + 1.0


class RotaryEncoding(PositionEncoding):
    """Fused into the attention mixer's query/key preparation kernel through ``inv_freq``."""

    def __init__(self, head_dim: int, theta: float):
        if head_dim % 2:
            raise ValueError("rotary encoding needs an even head size")
        self.head_dim = int(head_dim)
        self.theta = float(theta)
        self.inv_freq: Optional[Tensor] = None

    def finalize(self, dtype: torch.dtype, device: torch.device) -> None:
        i = torch.arange(self.head_dim // 2, dtype=torch.float32)
        theta32 = torch.tensor(self.theta, dtype=torch.float32)
        inv = 1.0 / torch.pow(theta32, (2.0 * i) / float(self.head_dim))
        self.inv_freq = inv.to(device=device, dtype=torch.float32).contiguous()


class NoPositionEncoding(PositionEncoding):
    """Queries and keys are used as projected."""
    inv_freq = None

    def __init__(self, head_dim: int = 0):
        self.head_dim = int(head_dim)


register_position_encoding("rotary", RotaryEncoding)
register_position_encoding("none", NoPositionEncoding)
