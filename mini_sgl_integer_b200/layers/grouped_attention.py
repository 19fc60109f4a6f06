"""Softmax attention whose query heads share key heads, with an optional window and without positions in the scores.

q and k are divided by the root mean square over their whole projection (all heads at once); keys and values are cached in
pages per key head.  Projections as in layers/matrix_memory.py.
"""
from __future__ import annotations

from typing import List, Tuple

import torch

from ..kernel import float_ops as fo
from ..models.config import GroupedAttentionConfig
from .base import BaseOP, StateDict
from .float_linear import FloatLinear, take_f32


class GroupedAttention(BaseOP):
    def __init__(self, cfg: GroupedAttentionConfig, hidden: int, eps: float, dtype: torch.dtype, device):
        self._cfg, self._eps, self._device = cfg, eps, device
        self.o = FloatLinear(cfg.heads * cfg.vdim, [hidden], ["o"], dtype, device)

    def projections(self) -> List[Tuple[str, int]]:
        c = self._cfg
        return [("q", c.heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.kv_heads * c.vdim)]

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        c = self._cfg
        self.q_norm = take_f32(state_dict, prefix + "q.norm", (c.heads * c.dim,), self._device)
        self.k_norm = take_f32(state_dict, prefix + "k.norm", (c.kv_heads * c.dim,), self._device)
        self.o.load_state_dict(state_dict, prefix=prefix)

    def run(self, y: torch.Tensor, col: int, md, cache, index: int) -> torch.Tensor:
        """``y``: parts of the projections, this mixer's from column ``col`` on.  fp32 partial sums [parts, rows, hidden]."""
        c, T, dtype = self._cfg, y.shape[1], self.o.weight.dtype
        k, v = cache.k_cache(index), cache.v_cache(index)
        q = torch.empty((T, c.heads, fo.pad8(c.dim)), dtype=dtype, device=y.device)
        k_col = col + c.heads * c.dim
        fo.grouped_prepare(y, (col, k_col, k_col + c.kv_heads * c.dim), self.q_norm, self.k_norm, self._eps, md.out_loc, q, k, v, c.heads, c.kv_heads,
                           c.dim, c.vdim)
        out = fo.rows(T, c.heads * c.vdim, dtype, y.device)
        fo.grouped_attention(q, k, v, md.page_table, md.kv_lens, md.seq_start, out, c.kv_heads, c.dim, c.vdim, c.window or 0, c.scale, md.max_seqlen_q,
                             md.max_seqlen_k)
        return self.o.parts(out)
