"""Rotary position tables of the floating-point models: cos | sin, fp32 [positions, dims], built in 64-bit on the host.

Entry i of a rotated vector is paired with entry i + dims / 2; pair i turns by position * base^(-2 i / dims).  With a
YaRN ``scaling`` (factor, original, fast, slow) the slow pairs are divided by the factor, the fast ones are kept, a linear
ramp lies between, and cos and sin are multiplied by 0.1 ln(factor) + 1.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from ..models.config import RotarySpec


def rotary_frequencies(spec: RotarySpec) -> tuple[torch.Tensor, float]:
    """(float64 [dims / 2] angular frequencies, factor on cos and sin)."""
    half = spec.dims // 2
    i = torch.arange(half, dtype=torch.float64)
    freq = torch.pow(torch.tensor(float(spec.base), dtype=torch.float64), -i / half)
    if spec.scaling is None:
        return freq, 1.0
    y = spec.scaling

    def pair_with_turns(turns: float) -> float:          # (fractional) pair that makes `turns` turns in `original` positions
        return spec.dims * math.log(y.original / (turns * 2.0 * math.pi)) / (2.0 * math.log(spec.base))
    lo = max(math.floor(pair_with_turns(y.fast)), 0)
    hi = min(math.ceil(pair_with_turns(y.slow)), spec.dims - 1)
    slow_share = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq * (slow_share / y.factor + (1.0 - slow_share)), 0.1 * math.log(y.factor) + 1.0


def rotary_table(spec: Optional[RotarySpec], positions: int, device) -> Optional[torch.Tensor]:
    if spec is None or spec.dims == 0:
        return None
    freq, mult = rotary_frequencies(spec)
    ang = torch.arange(positions, dtype=torch.float64)[:, None] * freq[None, :]
    return (torch.cat((ang.cos(), ang.sin()), dim=1) * mult).to(torch.float32).to(device).contiguous()
