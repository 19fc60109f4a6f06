"""Latent attention: one latent and one rotated key part per token, shared by all heads, is all that is cached.

Per head the score is (q_n . W_uk c + q_r . k_r) * scale and the value W_uv c.  Here the queries are taken into the latent
space instead (q_n W_uk, a per-head linear), the heads attend to the cached rows (c | k_r) directly, and the averaged
latents are multiplied by W_uv afterwards: keys and values are never expanded, for prompts and decoding alike.
A layer with ``kv_from`` has no key projection and reads the other layer's rows.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernel import float_ops as fo
from ..models.config import LatentAttentionConfig
from .base import BaseOP, StateDict
from .float_linear import FloatLinear, padded_rows, take, take_f32


class LatentAttention(BaseOP):
    def __init__(self, cfg: LatentAttentionConfig, hidden: int, layer_id: int, norm_eps: float, rope: Optional[torch.Tensor],
                 dtype: torch.dtype, device):
        self._cfg, self._eps, self._rope = cfg, norm_eps, rope
        self._cache_layer = layer_id if cfg.kv_from is None else cfg.kv_from
        self._dtype, self._device = dtype, device
        outs, names = [cfg.heads * (cfg.dim + cfg.rot_dim)], ["q"]
        if cfg.kv_from is None:
            outs.append(cfg.kv_rank + cfg.rot_dim)
            names.append("dkv")
        self.qd = FloatLinear(hidden, outs, names, dtype, device)
        self.o = FloatLinear(cfg.heads * cfg.vdim, [hidden], ["o"], dtype, device)
        self.dkv_norm: Optional[torch.Tensor] = None

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        c = self._cfg
        self.qd.load_state_dict(state_dict, prefix=prefix)
        self.o.load_state_dict(state_dict, prefix=prefix)
        if c.kv_from is None:
            self.dkv_norm = take_f32(state_dict, prefix + "dkv.norm", (c.kv_rank,), self._device)
        uk = take(state_dict, prefix + "uk", (c.heads * c.dim, c.kv_rank)).view(c.heads, c.dim, c.kv_rank)
        self.uk = padded_rows(uk.to(self._device).transpose(1, 2), self._dtype, self._device)             # [heads, kv_rank, dim]
        uv = take(state_dict, prefix + "uv", (c.heads * c.vdim, c.kv_rank)).view(c.heads, c.vdim, c.kv_rank)
        self.uv = padded_rows(uv, self._dtype, self._device)                                              # [heads, vdim, kv_rank]
        self.sink = take_f32(state_dict, prefix + "sink", (c.heads,), self._device)

    def forward(self, x: torch.Tensor, md, cache) -> torch.Tensor:
        c, T = self._cfg, x.shape[0]
        lat = fo.pad8(c.kv_rank + c.rot_dim)
        new = lambda n: torch.empty((T, c.heads, n), dtype=x.dtype, device=x.device)
        qn, q_lat, o_lat = new(fo.pad8(c.dim)), new(lat), new(fo.pad8(c.kv_rank))
        rows = cache.k_cache(self._cache_layer)
        fo.latent_prepare(self.qd.parts(x), md.positions, md.out_loc, self._rope, self.dkv_norm, self._eps, qn, q_lat,
                          rows if c.kv_from is None else None, c.heads, c.dim, c.rot_dim, c.kv_rank)
        fo.head_linear(qn[..., :c.dim], self.uk, q_lat[..., :c.kv_rank])
        fo.latent_attention(q_lat, rows, md.page_table, md.kv_lens, md.seq_start, self.sink, o_lat, c.kv_rank, c.rot_dim,
                            c.window or 0, c.scale, md.max_seqlen_q, md.max_seqlen_k)
        heads = fo.rows(T, c.heads * c.vdim, x.dtype, x.device)
        fo.head_linear(o_lat[..., :c.kv_rank], self.uv, heads.as_strided((T, c.heads, c.vdim), (heads.stride(0), c.vdim, 1)))
        return self.o.parts(heads)
