"""Next tokens from logits (engine/sample.py:74): greedy, on the device, the lowest index winning ties."""
from __future__ import annotations

import torch


def greedy(logits: torch.Tensor) -> torch.Tensor:
    """int32 [rows] from fp32 logits or the integer model's Q15.16 ones."""
    if logits.dtype == torch.int32:
        from ..models.qwen3_integer import argmax_int32
        return argmax_int32(logits)
    from ..kernel.float_ops import argmax_f32
    return argmax_f32(logits)
