"""Recurrent mixers with a matrix per head as state (S [dim, vdim], fp32), written by k w^T and read by S^T q.

Each class lists its input projections (``projections``) and works on their stacked output from a given column on
(``run``), so that one linear can serve several mixers that read the same input (layers/projected.py).
"""
from __future__ import annotations

from typing import List, Tuple

import torch

from ..kernel import float_ops as fo
from ..models.config import GatedDeltaConfig, MLSTMConfig, Mamba2Config
from .base import BaseOP, StateDict
from .float_linear import FloatLinear, take, take_f32


class MatrixMemory(BaseOP):
    """What the three kinds share: preparation, scan and output kernels around one layout of columns."""

    kind: int
    gate: int

    def __init__(self, heads: int, qk_heads: int, dim: int, vdim: int, hidden: int, eps: float, dtype: torch.dtype, device):
        self._heads, self._qk, self._dim, self._vdim, self._eps, self._device = heads, qk_heads, dim, vdim, eps, device
        self._q_scale, self._cap, self._group = 1.0, 0.0, vdim
        self._conv_w = self._conv_b = self._skip = None
        self.o = FloatLinear(heads * vdim, [hidden], ["o"], dtype, device)

    def projections(self) -> List[Tuple[str, int]]:
        raise NotImplementedError

    def _layout(self, order: str, first: int, gate_cols: Tuple[int, int], out_gate: int) -> None:
        """``order`` of the q, k and v columns, which begin at ``first``; the columns of the gates."""
        d, v = (self._qk * self._dim, self._dim), (self._heads * self._vdim, self._vdim)
        self._segments = [v if c == "v" else d for c in order]
        at, start = {}, 0
        for c, (w, h) in zip(order, self._segments):
            at[c] = start
            start += w // h * fo.pad8(h)
        self._row, self._offsets = start, (at["q"], at["k"], at["v"])
        self._first, self._gate_cols, self._out_gate = first, gate_cols, out_gate

    def run(self, y: torch.Tensor, col: int, md, cache, index: int) -> torch.Tensor:
        """``y``: parts of the projections, this mixer's from column ``col`` on.  fp32 partial sums [parts, rows, hidden]."""
        T, dev, dtype, H = y.shape[1], y.device, self.o.weight.dtype, self._heads
        f32 = lambda *s: torch.empty(s, dtype=torch.float32, device=dev)
        exp = self.kind == fo.MEMORY_EXP
        taps = 0 if self._conv_w is None else self._conv_w.shape[1]
        n = cache.state(index, "n") if exp else None
        rows, gates, o, den = fo.rows(T, self._row, dtype, dev), f32(T, H, 4), f32(T, H * self._vdim), f32(T, H) if exp else None
        fo.memory_prepare(y, col + self._first, self._segments, self._conv_w, self._conv_b, cache.state(index, "conv") if taps > 1 else None, md.slots,
                          md.positions, md.seq_start, md.seq_ids, rows, self.kind, H, [col + c for c in self._gate_cols], self.gate_a, self.gate_b,
                          gates, self._cap, n)
        fo.memory_scan(rows, self._offsets, self._qk, H, self._dim, self._vdim, self.kind, gates, self._q_scale, self._skip,
                       cache.state(index, "S"), n, md.slots, md.positions, md.seq_start, o, den,
                       md.max_seqlen_q)
        out = fo.rows(T, H * self._vdim, dtype, dev)
        fo.memory_output(o, den, H, self._vdim, self._group, y, col + self._out_gate, self.gate, self.norm, self._eps, out)
        return self.o.parts(out)


class MLSTM(MatrixMemory):
    """S_t = e^f S_(t-1) + e^i k v^T with log gates cap * tanh((W x + b) / cap) (f through logsigmoid), read out as S^T q divided
    by max(|n . q|, 1) of the same recurrence without v; everything relative to a running maximum of the exponents.
    Heads normed, times a gain over all of them, times sigmoid(W_g x)."""

    kind, gate = fo.MEMORY_EXP, fo.GATE_SIGMOID_AFTER

    def __init__(self, cfg: MLSTMConfig, hidden: int, eps: float, dtype: torch.dtype, device):
        super().__init__(cfg.heads, cfg.heads, cfg.dim, cfg.vdim, hidden, eps, dtype, device)
        self._q_scale, self._cap = cfg.dim ** -0.5, cfg.gate_cap
        d, v, h = cfg.heads * cfg.dim, cfg.heads * cfg.vdim, cfg.heads
        self._layout("qkv", 0, (2 * d + 2 * v, 2 * d + 2 * v + h), 2 * d + v)

    def projections(self):
        d, v, h = self._heads * self._dim, self._heads * self._vdim, self._heads
        return [("q", d), ("k", d), ("v", v), ("g", v), ("f", h), ("i", h)]

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        vec = lambda name, n: take_f32(state_dict, prefix + name, (n,), self._device)
        self.gate_a, self.gate_b = vec("f.b", self._heads), vec("i.b", self._heads)
        self.norm = vec("norm", self._heads * self._vdim)
        self.o.load_state_dict(state_dict, prefix=prefix)


class GatedDelta(MatrixMemory):
    """S <- g S, S <- S + k (beta (v - S^T k))^T: the value that the memory returns for k moves towards v by beta.  q, k and v
    pass short convolutions with silu, q and k are unit vectors.  Heads normed with one gain for all, times silu(W_g x)."""

    kind, gate = fo.MEMORY_DELTA, fo.GATE_SILU_AFTER

    def __init__(self, cfg: GatedDeltaConfig, hidden: int, eps: float, dtype: torch.dtype, device):
        super().__init__(cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim, hidden, eps, dtype, device)
        self._q_scale, self._taps = cfg.dim ** -0.5, cfg.conv
        d, v, h = cfg.kv_heads * cfg.dim, cfg.heads * cfg.vdim, cfg.heads
        self._layout("qkv", 0, (2 * d + 2 * v, 2 * d + 2 * v + h), 2 * d + v)

    def projections(self):
        d, v, h = self._qk * self._dim, self._heads * self._vdim, self._heads
        return [("q", d), ("k", d), ("v", v), ("g", v), ("a", h), ("b", h)]

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        vec = lambda name, n: take_f32(state_dict, prefix + name, (n,), self._device)
        self.gate_a, self.gate_b, self.norm = vec("A_log", self._heads), vec("dt_bias", self._heads), vec("norm", self._vdim)
        widths = [self._qk * self._dim, self._qk * self._dim, self._heads * self._vdim]
        self._conv_w = torch.cat([take_f32(state_dict, f"{prefix}{c}.conv", (n, self._taps), self._device) for c, n in zip("qkv", widths)]).contiguous()
        self.o.load_state_dict(state_dict, prefix=prefix)


class Mamba2(MatrixMemory):
    """S_t = exp(-e^A dt) S_(t-1) + dt B x^T, y = S^T C + D x, dt = softplus(pre + bias); x, B and C pass one short convolution
    with bias and silu; times silu(z), then normed in equal parts."""

    kind, gate = fo.MEMORY_SSD, fo.GATE_SILU_BEFORE

    def __init__(self, cfg: Mamba2Config, hidden: int, eps: float, dtype: torch.dtype, device):
        super().__init__(cfg.heads, cfg.groups, cfg.state, cfg.vdim, hidden, eps, dtype, device)
        self._group, self._taps = cfg.inner // cfg.norm_groups, cfg.conv
        self._channels = cfg.inner + 2 * cfg.groups * cfg.state
        dt = cfg.inner + self._channels
        self._layout("vkq", cfg.inner, (dt, dt), 0)

    def projections(self):
        return [("in", self._heads * self._vdim + self._channels + self._heads)]

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        vec = lambda name, n: take_f32(state_dict, prefix + name, (n,), self._device)
        self.gate_a, self.gate_b, self._skip = (vec(n, self._heads) for n in ("A_log", "dt_bias", "D"))
        self.norm = vec("norm", self._heads * self._vdim)
        self._conv_w = take(state_dict, prefix + "conv", (self._channels, self._taps)).to(device=self._device, dtype=torch.float32).contiguous()
        self._conv_b = vec("conv.b", self._channels)
        self.o.load_state_dict(state_dict, prefix=prefix)
