"""One linear in front of one or more mixers that read the same input."""
from __future__ import annotations

from typing import List, Sequence, Tuple

import torch

from .base import BaseOP, StateDict
from .float_linear import FloatLinear


class ProjectedMixers(BaseOP):
    """``sides``: (prefix of its tensors, mixer).  A mixer lists its projections and continues from their output."""

    def __init__(self, hidden: int, sides: Sequence[Tuple[str, BaseOP]], dtype: torch.dtype, device):
        self._sides, self._cols = list(sides), []
        names, sizes = [], []
        for prefix, mixer in sides:
            self._cols.append(sum(sizes))
            for name, n in mixer.projections():
                names.append(prefix + name)
                sizes.append(n)
        self.proj = FloatLinear(hidden, sizes, names, dtype, device, pad_out=8)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        self.proj.load_state_dict(state_dict, prefix=prefix)
        for side, mixer in self._sides:
            mixer.load_state_dict(state_dict, prefix=prefix + side)

    def forward(self, x: torch.Tensor, md, cache, index: int) -> List[torch.Tensor]:
        """Per mixer fp32 partial sums [parts, rows, hidden]; ``index``: the run whose cache and state are used."""
        y = self.proj.parts(x)
        return [mixer.run(y, col, md, cache, index) for (_, mixer), col in zip(self._sides, self._cols)]
