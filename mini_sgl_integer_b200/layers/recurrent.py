"""Recurrent mixers over a per-sequence fp32 state."""
from __future__ import annotations

import torch

from ..kernel import float_ops as fo
from ..models.config import MinGRUConfig
from .base import BaseOP, StateDict
from .float_linear import FloatLinear, take_f32


class MinGRU(BaseOP):
    """S_t = (1 - z) S_(t-1) + z c with z = sigmoid(W_z x + b_z) and c = g(W_x x + b_x), g(u) = u + 1/2 for u >= 0 and
    sigmoid(u) below; output W_o (S_t * silu(W_g x)).  The three projections are one linear."""

    def __init__(self, cfg: MinGRUConfig, hidden: int, state_index: int, dtype: torch.dtype, device):
        self._width, self._state_index, self._device = cfg.width, state_index, device
        self.zug = FloatLinear(hidden, [cfg.width] * 3, ["z", "x", "g"], dtype, device)
        self.o = FloatLinear(cfg.width, [hidden], ["o"], dtype, device)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        self.zug.load_state_dict(state_dict, prefix=prefix)
        self.o.load_state_dict(state_dict, prefix=prefix)
        self.bias_z = take_f32(state_dict, prefix + "z.b", (self._width,), self._device)
        self.bias_u = take_f32(state_dict, prefix + "x.b", (self._width,), self._device)

    def forward(self, x: torch.Tensor, md, cache) -> torch.Tensor:
        y = fo.rows(x.shape[0], self._width, x.dtype, x.device)
        fo.mingru(self.zug.parts(x), self.bias_z, self.bias_u, cache.state(self._state_index), md.slots, md.positions, md.seq_start,
                  md.kv_lens.numel(), y)
        return self.o.parts(y)
