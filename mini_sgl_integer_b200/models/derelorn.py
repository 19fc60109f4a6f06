"""Derelorn: a decoder of matrix memories, with a layer type that runs attention and a state-space memory side by side.

    x = norm(embed[token])
    a run of a layer:  x <- x + norm1b(mixer(norm1 x));  x <- x + norm2b(mlp(norm2 x))
    logits = head norm(x)

Layers start .. stop - 1 may run several times with the same weights; a vector of its own is added to x in front of each pass,
and every run has its own cache and state.  The stream x is fp32 and updated in place; a sublayer's last linear stays a
stack of partial sums, and one kernel finishes it: output norm, residual add, the vector of a pass that begins, and the
norm in front of the next linear, whose result is in the model's dtype.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from ..kernel import float_ops as fo
from ..layers.base import BaseOP, OPList, StateDict
from ..layers.float_linear import FloatLinear, GatedSiluMLP, take, take_f32
from ..layers.grouped_attention import GroupedAttention
from ..layers.matrix_memory import GatedDelta, MLSTM, Mamba2
from ..layers.projected import ProjectedMixers
from .config import DerelornConfig, HybridLayerConfig
from .hybrid import HybridForCausalLM

After = Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]       # the vector to add and the norm in front of what follows


class DerelornLayer(BaseOP):
    def __init__(self, config: DerelornConfig, layer: HybridLayerConfig, dtype: torch.dtype, device):
        hidden, m = config.hidden_size, layer.mixer
        self._hidden, self._eps, self._device = hidden, config.norm_eps, device
        args = (hidden, config.norm_eps, dtype, device)
        self._parallel = layer.type == "parallel"
        if self._parallel:
            sides = [("left.", GroupedAttention(m.left, *args)), ("right.", Mamba2(m.right, *args))]
        else:
            sides = [("", MLSTM(m, *args) if layer.type == "mlstm" else GatedDelta(m, *args))]
        self.mix = ProjectedMixers(hidden, sides, dtype, device)
        self.mlp: Optional[GatedSiluMLP] = GatedSiluMLP(hidden, layer.mlp.ff, dtype, device) if layer.mlp is not None else None

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        gain = lambda name: take_f32(state_dict, prefix + name, (self._hidden,), self._device)
        self.norm1, self.norm1b = gain("norm1"), gain("norm1b")
        self.mix.load_state_dict(state_dict, prefix=prefix + "mix.")
        if self._parallel:
            self.left_out, self.right_out = gain("mix.left.out"), gain("mix.right.out")
        if self.mlp is not None:
            self.norm2, self.norm2b = gain("norm2"), gain("norm2b")
            self.mlp.load_state_dict(state_dict, prefix=prefix + "mlp.")
        else:
            for name in ("norm2", "norm2b"):
                state_dict.pop(prefix + name, None)            # gains without a sublayer have nothing to act on

    def forward(self, x: torch.Tensor, xt: torch.Tensor, md, cache, index: int, after: After, keep: bool) -> None:
        """``x`` (fp32) is the stream, ``xt`` its norm1; afterwards ``xt`` holds what ``after`` asks for.  ``keep``: x is needed
        afterwards."""
        ys = self.mix.forward(xt, md, cache, index)
        mean = (self.left_out, ys[1], self.right_out) if self._parallel else None
        end = dict(add=after[0], final_w=after[1])
        out = x if keep else None
        if self.mlp is None:
            fo.sublayer_end(ys[0], x, self.norm1b, self._eps, out, xt, xt.dtype, mean_with=mean, **end)
        else:
            fo.sublayer_end(ys[0], x, self.norm1b, self._eps, x, xt, xt.dtype, mean_with=mean, final_w=self.norm2)
            fo.sublayer_end(self.mlp.forward(xt), x, self.norm2b, self._eps, out, xt, xt.dtype, **end)


class DerelornForCausalLM(HybridForCausalLM):
    def __init__(self, config: DerelornConfig, dtype: torch.dtype = torch.bfloat16, device="cuda"):
        self._config, self._dtype, self._device = config, dtype, torch.device(device)
        fo.dtype_code(dtype)
        self._runs = config.runs
        self.layers = OPList([DerelornLayer(config, l, dtype, self._device) for l in config.layers])
        self.head = FloatLinear(config.hidden_size, [config.vocab_size], ["head"], dtype, self._device)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        c = self._config
        gain = lambda name: take_f32(state_dict, prefix + name, (c.hidden_size,), self._device)
        self.embed = take(state_dict, prefix + "embed", (c.vocab_size, c.hidden_size)).to(device=self._device, dtype=self._dtype).contiguous()
        self.embed_norm, self.final_norm = gain("embed.norm"), gain("final.norm")
        self.loop_step = take_f32(state_dict, prefix + "loop.step", (c.loop.times, c.hidden_size), self._device) if c.loop is not None else None
        for i, layer in enumerate(self.layers.op_list):
            layer.load_state_dict(state_dict, prefix=f"{prefix}l{i}.", _internal=True)
        self.head.load_state_dict(state_dict, prefix=prefix)
        if not _internal and state_dict:
            raise RuntimeError(f"Unexpected keys in state_dict: {list(state_dict.keys())}")

    def _before(self, k: int) -> After:
        """The vector added in front of run ``k`` and the norm that its mixer reads; behind the last run, the final norm."""
        if k == len(self._runs):
            return None, self.final_norm
        r = self._runs[k]
        return None if r.begins is None else self.loop_step[r.begins], self.layers.op_list[r.layer].norm1

    def forward_tokens(self, ids: torch.Tensor, md, cache, logit_rows: Optional[torch.Tensor] = None,
                       trace: Optional[List[torch.Tensor]] = None) -> Optional[torch.Tensor]:
        """fp32 logits [rows, vocab] of the token rows ``logit_rows`` (all rows when None; None for an empty selection).
        ``trace`` receives a copy of the stream that leaves every run of a layer."""
        c, T, eps = self._config, ids.numel(), self._config.norm_eps
        x = torch.empty((T, c.hidden_size), dtype=torch.float32, device=self._device)
        first = torch.empty((1, T, c.hidden_size), dtype=torch.float32, device=self._device)
        xt_buf = torch.empty((T, fo.pad8(c.hidden_size)), dtype=self._dtype, device=self._device)
        xt = xt_buf[:, :c.hidden_size]
        fo.embed_bigram(self.embed, None, ids, md.positions, md.seq_ids, md.seq_start, md.slots, None, 0, 0, 0, first[0], None)
        add, norm = self._before(0)
        fo.sublayer_end(first, None, self.embed_norm, eps, x, xt, self._dtype, add=add, final_w=norm)
        for k, r in enumerate(self._runs):
            after = self._before(k + 1)
            layer = self.layers.op_list[r.layer]
            if trace is None:
                layer.forward(x, xt, md, cache, k, after, k + 1 < len(self._runs))
            else:
                layer.forward(x, xt, md, cache, k, (None, None), True)
                trace.append(x.clone())
                fo.sublayer_end(None, x, None, eps, x, xt, self._dtype, add=after[0], final_w=after[1])
        if logit_rows is not None:
            if logit_rows.numel() == 0:
                return None
            xt = xt_buf.index_select(0, logit_rows)[:, :c.hidden_size]
        return self.head.forward(xt, out_f32=True)


def random_weights(config: DerelornConfig, seed: int, device="cpu", dtype: torch.dtype = torch.bfloat16) -> StateDict:
    """Seeded random weights under the checkpoint's names, scaled so that streams keep a moderate size."""
    dev = torch.device(device)
    g = torch.Generator(device=dev).manual_seed(seed)
    rnd = lambda *s: torch.randn(s, generator=g, device=dev)
    mat = lambda n, k: (rnd(n, k) * k ** -0.5).to(dtype)
    gain = lambda n: (1.0 + 0.2 * rnd(n)).to(dtype)
    vec = lambda n, mean=0.0, size=1.0: (mean + size * rnd(n)).to(dtype)
    W = config.hidden_size
    sd: StateDict = {"embed": rnd(config.vocab_size, W).to(dtype), "embed.norm": gain(W)}
    if config.loop is not None:
        sd["loop.step"] = (0.5 * rnd(config.loop.times, W)).to(dtype)
    for i, l in enumerate(config.layers):
        p, m, mix = f"l{i}.", l.mixer, f"l{i}.mix."
        sd[p + "norm1"], sd[p + "norm1b"] = gain(W), gain(W)
        if l.type == "parallel":
            a, s = m.left, m.right
            for name, n in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                sd[f"{mix}left.{name}"] = mat(n, W)
            sd[mix + "left.q.norm"], sd[mix + "left.k.norm"], sd[mix + "left.o"] = gain(a.heads * a.dim), gain(a.kv_heads * a.dim), mat(W, a.heads * a.vdim)
            channels = s.inner + 2 * s.groups * s.state
            sd[mix + "right.in"] = mat(s.inner + channels + s.heads, W)
            sd[mix + "right.conv"], sd[mix + "right.conv.b"] = mat(channels, s.conv), vec(channels, size=0.3)
            sd[mix + "right.dt_bias"], sd[mix + "right.A_log"], sd[mix + "right.D"] = vec(s.heads, -3.0), vec(s.heads, 0.5), vec(s.heads, 1.0, 0.3)
            sd[mix + "right.norm"], sd[mix + "right.o"] = gain(s.inner), mat(W, s.inner)
            sd[mix + "left.out"], sd[mix + "right.out"] = gain(W), gain(W)
        else:
            qk, v = (m.heads if l.type == "mlstm" else m.kv_heads) * m.dim, m.heads * m.vdim
            for name, n in (("q", qk), ("k", qk), ("v", v), ("g", v)):
                sd[mix + name] = mat(n, W)
            sd[mix + "o"] = mat(W, v)
            if l.type == "mlstm":
                for name, mean in (("i", -1.0), ("f", 4.0)):
                    sd[mix + name], sd[f"{mix}{name}.b"] = mat(m.heads, W), vec(m.heads, mean)
                sd[mix + "norm"] = gain(v)
            else:
                for name, n in (("q", qk), ("k", qk), ("v", v)):
                    sd[f"{mix}{name}.conv"] = mat(n, m.conv)
                sd[mix + "a"], sd[mix + "b"] = mat(m.heads, W), mat(m.heads, W)
                sd[mix + "A_log"], sd[mix + "dt_bias"], sd[mix + "norm"] = vec(m.heads, 0.5), vec(m.heads, -4.0), gain(m.vdim)
        if l.mlp is not None:
            sd[p + "norm2"], sd[p + "norm2b"] = gain(W), gain(W)
            sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"] = mat(l.mlp.ff, W), mat(l.mlp.ff, W), mat(W, l.mlp.ff)
    sd["final.norm"], sd["head"] = gain(W), mat(config.vocab_size, W)
    return sd
