"""Device memory of a hybrid model: per attention layer pools of 16-token pages of cached rows, per recurrent layer fp32
states of every sequence, and each sequence's last token.

    planes dtype [pages, 16, heads * pitch]   keys (or latent | rotated key part), values; pitch a multiple of 8 values
    state  fp32  [slots, ...]                 read as zero when a sequence starts, so a slot needs no clearing
    prev   int32 [slots]

``config.memory`` says what each layer (each run of a layer, where layers run several times) keeps.  One more page and slot
than asked for are allocated: padding rows of captured decode batches live there.
"""
from __future__ import annotations

import torch

from ..kernel.float_ops import pad8
from . import BaseKVCache

PAGE_SIZE = 16


class HybridCache(BaseKVCache):
    def __init__(self, config, num_pages: int, num_slots: int, dtype: torch.dtype, device) -> None:
        """``config.memory``: a ``RunMemory`` per run."""
        self._device, self._dtype = torch.device(device), dtype
        if self._device.type != "cuda":
            raise RuntimeError("the cache lives in GPU memory; there is no CPU fallback")
        self.num_pages, self.num_slots, self._memory = num_pages, num_slots, config.memory
        self.spare_page, self.spare_slot = num_pages, num_slots
        zeros = lambda shape, t: torch.zeros(shape, dtype=t, device=self._device)
        self._planes = {i: [zeros((num_pages + 1, PAGE_SIZE, h * pad8(n)), dtype) for h, n in m.planes] for i, m in enumerate(self._memory) if m.planes}
        self._state = {(i, name): zeros((num_slots + 1, *shape), torch.float32) for i, m in enumerate(self._memory) for name, shape in m.state}
        self.prev_tokens = zeros(num_slots + 1, torch.int32)

    @staticmethod
    def page_bytes(config, dtype: torch.dtype) -> int:
        """Bytes of one page over all layers."""
        return sum(PAGE_SIZE * h * pad8(n) * dtype.itemsize for m in config.memory for h, n in m.planes)

    @staticmethod
    def slot_bytes(config) -> int:
        """Bytes of one sequence's states over all layers."""
        count = 0
        for m in config.memory:
            for _, shape in m.state:
                n = 4
                for d in shape:
                    n *= d
                count += n
        return count

    def k_cache(self, index: int) -> torch.Tensor:
        return self._planes[index][0]

    def v_cache(self, index: int) -> torch.Tensor:
        prefix = self._memory[index].value_prefix
        return self._planes[index][1] if prefix is None else self._planes[index][0][..., :prefix]

    def state(self, index: int, name: str = "s") -> torch.Tensor:
        return self._state[index, name]

    def store_kv(self, k: torch.Tensor, v: torch.Tensor, out_loc: torch.Tensor, layer_id: int) -> None:
        """Rows [tokens, heads * values] to token locations.  Where the value is a part of the key row, ``v`` is not stored
        again.  The models' own forward stores from its preparation kernels."""
        m, loc = self._memory[layer_id], out_loc.to(torch.int64)
        for (h, n), plane, rows in zip(m.planes, self._planes[layer_id], (k, v)):
            plane.view(-1, h, pad8(n))[loc, :, :n] = rows.reshape(-1, h, n).to(self._dtype)

    @property
    def device(self) -> torch.device:
        return self._device

    @property
    def dtype(self) -> torch.dtype:
        return self._dtype

    @property
    def num_layers(self) -> int:
        return len(self._memory)
