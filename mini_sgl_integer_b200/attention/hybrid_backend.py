"""Backend of hybrid models (paged attention + recurrent state): the metadata of a batch and its CUDA-graph buffers,
behind the interface of ``BaseAttnBackend``.  The mixers launch their own kernels with this metadata, so there is no
per-layer ``forward`` on separate q, k and v."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from .backend import BaseAttnBackend, BaseAttnMetadata

PAGE_SIZE = 16


@dataclass
class HybridMetadata(BaseAttnMetadata):
    positions: torch.Tensor               # int32 [tokens]
    out_loc: torch.Tensor                 # int32 [tokens] cache rows (page * 16 + offset) of the new tokens
    page_table: torch.Tensor              # int32 [bs, pitch]
    kv_lens: torch.Tensor                 # int32 [bs] keys per request including the new tokens
    slots: torch.Tensor                   # int32 [bs] rows of the recurrent state
    seq_start: Optional[torch.Tensor]     # int32 [bs + 1] first token of each request; None: one new token each (decode)
    seq_ids: Optional[torch.Tensor]       # int32 [tokens]
    max_seqlen_q: int
    max_seqlen_k: int

    def get_last_indices(self, bs: int) -> torch.Tensor:
        if self.seq_start is not None:
            return self.seq_start[1: 1 + bs] - 1
        return torch.arange(bs, device=self.kv_lens.device)


class B200HybridBackend(BaseAttnBackend):
    def __init__(self, config, kvcache, page_table: Optional[torch.Tensor] = None) -> None:
        self.config, self.kvcache, self.device = config, kvcache, kvcache.device
        self._page_table = page_table
        self.capture_bs: List[int] = []
        self.max_seq_len = 0
        self._cap: Optional[dict] = None

    @property
    def page_table(self) -> torch.Tensor:
        if self._page_table is not None:
            return self._page_table
        from ..core import get_global_ctx
        return get_global_ctx().page_table

    def forward(self, q, k, v, layer_id, batch):
        raise NotImplementedError("the mixers of hybrid models run their attention inside their layers")

    def prepare_metadata(self, batch) -> None:
        """From ``batch.padded_reqs`` (table_idx, cached_len, device_len), ``batch.positions`` and ``batch.out_loc``."""
        reqs = batch.padded_reqs
        bs = len(reqs)
        q_lens = torch.tensor([r.device_len - r.cached_len for r in reqs])
        tokens = int(q_lens.sum())
        # one host array, one copy: slots | kv_lens | seq_start (bs + 1) | seq_ids
        host = torch.zeros(3 * bs + 1 + tokens, dtype=torch.int32)
        host[:bs] = torch.tensor([r.table_idx for r in reqs], dtype=torch.int32)
        host[bs:2 * bs] = torch.tensor([r.device_len for r in reqs], dtype=torch.int32)
        host[2 * bs + 1:3 * bs + 1] = q_lens.cumsum(0)
        host[3 * bs + 1:] = torch.repeat_interleave(torch.arange(bs, dtype=torch.int32), q_lens)
        dev = host.pin_memory().to(self.device, non_blocking=True)
        # (the kernels take plain pointers: pieces of one int32 array are aligned enough)
        slots, kv_lens, start, seq = torch.split(dev, [bs, bs, bs + 1, tokens])
        table = self.page_table.index_select(0, slots)
        decode = batch.is_decode
        batch.attn_metadata = HybridMetadata(batch.positions, batch.out_loc, table, kv_lens, slots, None if decode else start,
                                             None if decode else seq, int(q_lens.max()), max(r.device_len for r in reqs))

    # ------------------------------------------------------------------ CUDA graphs (decode only)
    def init_capture_graph(self, max_seq_len: int, bs_list: List[int]) -> None:
        if self._cap is not None:
            raise RuntimeError("capture buffers already initialised")
        self.max_seq_len, self.capture_bs = int(max_seq_len), sorted(bs_list)
        n, pitch = max(bs_list), self.page_table.shape[1]
        full = lambda v, *s: torch.full(s, v, dtype=torch.int32, device=self.device)
        self._cap = {"page_table": full(self.kvcache.spare_page, n, pitch), "kv_lens": full(1, n), "slots": full(self.kvcache.spare_slot, n)}

    def prepare_for_capture(self, batch) -> None:
        bs = batch.size
        if self._cap is None or bs not in self.capture_bs:
            raise RuntimeError(f"batch size {bs} was not registered with init_capture_graph")
        if not batch.is_decode:
            raise RuntimeError("CUDA graph capture only supports decode")
        c = {k: v[:bs] for k, v in self._cap.items()}
        batch.attn_metadata = HybridMetadata(batch.positions, batch.out_loc, c["page_table"], c["kv_lens"], c["slots"], None, None, 1,
                                             self.max_seq_len)

    def prepare_for_replay(self, batch) -> None:
        md, bs = batch.attn_metadata, batch.padded_size
        if self._cap is None or not isinstance(md, HybridMetadata) or bs not in self.capture_bs:
            raise RuntimeError("prepare_metadata must run first, for a registered batch size")
        for name, buf in self._cap.items():
            buf[:bs].copy_(getattr(md, name))
