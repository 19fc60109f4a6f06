"""Linear layers of the floating-point models: a weight [out, in] kept in the model's dtype with rows padded to a pitch
of 8 values (what TMA wants), applied by the kernels of kernel/float_ops.py."""
from __future__ import annotations

import math
from typing import Sequence

import torch

from ..kernel import float_ops as fo
from .base import BaseOP, StateDict


def take(state_dict: StateDict, key: str, shape: Sequence[int]) -> torch.Tensor:
    """Pops a tensor of the given shape."""
    if key not in state_dict:
        raise KeyError(f"missing key in state_dict: {key}")
    item = state_dict.pop(key)
    if tuple(item.shape) != tuple(shape):
        raise ValueError(f"Shape mismatch for {key}: {tuple(shape)} vs {tuple(item.shape)}")
    return item


def take_f32(state_dict: StateDict, key: str, shape: Sequence[int], device) -> torch.Tensor:
    """A vector that the kernels read in 32-bit (norm gains, biases, coefficients)."""
    return take(state_dict, key, shape).to(device=device, dtype=torch.float32).contiguous()


def padded_rows(w: torch.Tensor, dtype: torch.dtype, device) -> torch.Tensor:
    """``w`` [.., n, k] on the device in ``dtype`` with a row pitch that is a multiple of 8 values."""
    k = w.shape[-1]
    if k % 8 == 0:
        return w.to(device=device, dtype=dtype).contiguous()
    buf = torch.zeros((*w.shape[:-1], fo.pad8(k)), dtype=dtype, device=device)
    buf[..., :k] = w.to(device=device, dtype=dtype)
    return buf[..., :k]


class FloatLinear(BaseOP):
    """W x without bias; ``weight`` may be several checkpoint tensors stacked along the output.  ``pad_out``: zero rows are
    added up to a multiple of it, so that the rows of the output start on aligned addresses."""

    def __init__(self, in_features: int, out_features: Sequence[int], names: Sequence[str], dtype: torch.dtype, device, pad_out: int = 1):
        self._in, self._outs, self._names, self._pad = in_features, tuple(out_features), tuple(names), -sum(out_features) % pad_out
        self._dtype, self._device = dtype, device
        self.weight = torch.empty(0)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        parts = [take(state_dict, prefix + n, (o, self._in)) for n, o in zip(self._names, self._outs)]
        if self._pad:
            parts.append(torch.zeros((self._pad, self._in), dtype=parts[0].dtype, device=parts[0].device))
        self.weight = padded_rows(parts[0] if len(parts) == 1 else torch.cat([p.to(self._device) for p in parts]), self._dtype, self._device)

    def forward(self, x: torch.Tensor, out_f32: bool = False) -> torch.Tensor:
        return fo.linear(x, self.weight, out_f32=out_f32)

    def parts(self, x: torch.Tensor) -> torch.Tensor:
        """The output as fp32 partial sums [parts, rows, out] for a kernel that adds them."""
        return fo.linear_parts(x, self.weight)


class XieluMLP(BaseOP):
    """down(act(up x)) with act = xIELU of the checkpoint's two numbers p, q: softplus(p) z^2 + z / 2 for z > 0,
    (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2 otherwise."""

    def __init__(self, hidden: int, ff: int, dtype: torch.dtype, device):
        self._ff = ff
        self.up = FloatLinear(hidden, [ff], ["up"], dtype, device)
        self.down = FloatLinear(ff, [hidden], ["down"], dtype, device)
        self._act = (0.0, 0.0)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        self.up.load_state_dict(state_dict, prefix=prefix)
        self.down.load_state_dict(state_dict, prefix=prefix)
        p, q = (float(v) for v in take(state_dict, prefix + "act", (2,)).to(torch.float64))
        softplus = lambda v: max(v, 0.0) + math.log1p(math.exp(-abs(v)))
        self._act = (softplus(p), 0.5 + softplus(q))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """fp32 partial sums [parts, rows, hidden]."""
        w = self.up.weight
        if fo.query("b200f_gemm_splits", x.shape[0], self._ff, x.shape[1], 1, fo.dtype_code(x.dtype)) == 1:
            act = fo.linear(x, w, act=fo.ACT_XIELU, act_a=self._act[0], act_b=self._act[1])     # in the linear's epilogue
        else:
            act = fo.rows(x.shape[0], self._ff, x.dtype, x.device)
            fo.xielu(self.up.parts(x), act, *self._act)
        return self.down.parts(act)


class GatedSiluMLP(BaseOP):
    """down(silu(gate x) * (up x)).  The rows of gate and up alternate in blocks of 16 (the last block filled up with zeros), so
    that both halves of a product meet in one accumulator tile of the linear."""

    BLOCK = 16

    def __init__(self, hidden: int, ff: int, dtype: torch.dtype, device):
        self._hidden, self._ff, self._dtype, self._device = hidden, ff, dtype, device
        self.weight = torch.empty(0)
        self.down = FloatLinear(ff, [hidden], ["down"], dtype, device)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        blocks = -(-self._ff // self.BLOCK)
        both = []
        for name in ("gate", "up"):
            w = take(state_dict, prefix + name, (self._ff, self._hidden)).to(self._device)
            fill = torch.zeros((blocks * self.BLOCK - self._ff, self._hidden), dtype=w.dtype, device=self._device)
            both.append(torch.cat([w, fill]).view(blocks, self.BLOCK, self._hidden))
        self.weight = padded_rows(torch.stack(both, dim=1).reshape(-1, self._hidden), self._dtype, self._device)
        self.down.load_state_dict(state_dict, prefix=prefix)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """fp32 partial sums [parts, rows, hidden]."""
        w, T = self.weight, x.shape[0]
        act = fo.rows(T, w.shape[0] // 2, x.dtype, x.device)
        if x.dtype == torch.bfloat16 and fo.query("b200f_gemm_splits", T, w.shape[0], x.shape[1], 1, fo.dtype_code(x.dtype)) == 1:
            fo.linear(x, w, out=act, act=fo.ACT_GATED_SILU)                                    # in the linear's epilogue
        else:
            fo.gated_silu(fo.linear_parts(x, w), act)
        return self.down.parts(act[:, :self._ff])
