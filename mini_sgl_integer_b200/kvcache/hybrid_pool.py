"""Device memory of a hybrid model: per attention layer a pool of 16-token pages of latent rows, per recurrent layer one
fp32 state vector per sequence, and each sequence's last token.

    rows   dtype [pages, 16, pitch]     (latent | rotated key part | zero padding), pitch a multiple of 8 values
    state  fp32  [slots, width]         read as zero when a sequence starts, so a slot needs no clearing
    prev   int32 [slots]

Layers that use another layer's cache have none of their own.  One more page and slot than asked for are allocated:
padding rows of captured decode batches live there.
"""
from __future__ import annotations

import torch

from ..kernel.float_ops import pad8
from . import BaseKVCache

PAGE_SIZE = 16


class HybridCache(BaseKVCache):
    def __init__(self, config, num_pages: int, num_slots: int, dtype: torch.dtype, device) -> None:
        """``config``: ``layers``, ``cache_layers`` and ``recurrent_layers`` of a hybrid model's configuration."""
        self._device, self._dtype = torch.device(device), dtype
        if self._device.type != "cuda":
            raise RuntimeError("the cache lives in GPU memory; there is no CPU fallback")
        self.num_pages, self.num_slots, self._num_layers = num_pages, num_slots, len(config.layers)
        self.spare_page, self.spare_slot = num_pages, num_slots
        self._rows, self._rank, self._state = {}, {}, {}
        for i in config.cache_layers:
            m = config.layers[i].mixer
            self._rank[i] = m.kv_rank
            self._rows[i] = torch.zeros((num_pages + 1, PAGE_SIZE, pad8(m.kv_rank + m.rot_dim)), dtype=dtype, device=self._device)
        for i in config.recurrent_layers:
            self._state[i] = torch.zeros((num_slots + 1, config.layers[i].mixer.width), dtype=torch.float32, device=self._device)
        self.prev_tokens = torch.zeros(num_slots + 1, dtype=torch.int32, device=self._device)

    @staticmethod
    def page_bytes(config, dtype: torch.dtype) -> int:
        """Bytes of one page over all layers."""
        return sum(PAGE_SIZE * pad8(config.layers[i].mixer.kv_rank + config.layers[i].mixer.rot_dim) * dtype.itemsize
                   for i in config.cache_layers)

    def k_cache(self, index: int) -> torch.Tensor:
        return self._rows[index]

    def v_cache(self, index: int) -> torch.Tensor:
        return self._rows[index][..., :self._rank[index]]

    def state(self, index: int) -> torch.Tensor:
        return self._state[index]

    def store_kv(self, k: torch.Tensor, v: torch.Tensor, out_loc: torch.Tensor, layer_id: int) -> None:
        """Rows (latent | rotated key part) to token locations; ``v`` is the latent part of the same rows and not stored
        twice.  The model's own forward stores from its preparation kernel."""
        rows = self._rows[layer_id].view(-1, self._rows[layer_id].shape[2])
        rows[out_loc.to(torch.int64), :k.shape[1]] = k.to(self._dtype)

    @property
    def device(self) -> torch.device:
        return self._device

    @property
    def dtype(self) -> torch.dtype:
        return self._dtype

    @property
    def num_layers(self) -> int:
        return self._num_layers
