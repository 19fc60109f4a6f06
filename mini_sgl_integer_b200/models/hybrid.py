"""What the floating-point model classes share: running the batch of the global context."""
from __future__ import annotations

from typing import Optional

import torch

from ..core import get_global_ctx
from ..kernel import float_ops as fo
from ..layers.base import BaseOP


class HybridForCausalLM(BaseOP):
    """A model with ``forward_tokens(ids, metadata, cache, logit_rows, trace)``, run with metadata that the "b200_hybrid"
    backend has prepared."""

    skips_empty_logits = True            # a batch whose ``logit_rows`` is empty runs without the head

    @property
    def config(self):
        return self._config

    def forward(self) -> Optional[torch.Tensor]:
        """Logits of the batch in the global context: of ``batch.logit_rows``, else of every request's last token."""
        ctx = get_global_ctx()
        batch = ctx.batch
        rows = batch.logit_rows
        if rows is None and batch.is_prefill:
            rows = batch.attn_metadata.get_last_indices(batch.size).to(torch.int64)
        return self.forward_tokens(batch.input_ids, batch.attn_metadata, ctx.attn_backend.kvcache, rows)

    check_status = staticmethod(fo.check_status)
