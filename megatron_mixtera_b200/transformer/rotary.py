"""Rotation tables: scaled cos / sin per position and pair, for kernels that rotate interleaved pairs."""
from __future__ import annotations

import math
from typing import Tuple

import torch

from .hybrid_config import RotaryConfig


def rotary_frequencies(rot: RotaryConfig) -> Tuple[torch.Tensor, float]:
    """(float64 frequency per pair, factor on cos and sin)."""
    i = torch.arange(rot.dims // 2, dtype=torch.float64)
    freq = rot.base ** (-2.0 * i / max(rot.dims, 1))
    sc = rot.scaling
    if sc is None:
        return freq, 1.0

    def index_of(turns: float) -> float:
        return rot.dims * math.log(sc.original / (2.0 * math.pi * turns)) / (2.0 * math.log(rot.base))

    lo = max(math.floor(index_of(sc.fast)), 0)
    hi = min(math.ceil(index_of(sc.slow)), rot.dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / sc.factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(sc.factor) + 1.0


def rotary_tables(rot: RotaryConfig, max_positions: int, device) -> Tuple[torch.Tensor, torch.Tensor]:
    """fp32 ``[max_positions, dims / 2]`` cos and sin; the angles are formed in float64 on the host."""
    freq, factor = rotary_frequencies(rot)
    angle = torch.outer(torch.arange(max_positions, dtype=torch.float64), freq)
    return tuple((f(angle) * factor).to(torch.float32).to(device).contiguous() for f in (torch.cos, torch.sin))
