"""Sefevik: a decoder of gated recurrences and latent attention with output norms and depth averages.

    x = X_0 = embed[token] (+ a bigram row of the previous and the current token)
    layer i:  x <- x + norm1(mixer(x));  x <- x + norm2(mlp(x));  X_(i+1) = x;  x <- sum_j dwa[j] X_j, j = 0 .. i + 1
    logits = head norm(x)

The stream x and every X_j are fp32; a copy of x in the model's dtype feeds the linears.  A sublayer's last linear stays
a stack of partial sums, and one kernel finishes it together with the norm, the residual add, the depth average and, at
the end of the model, the final norm (``sublayer_end``).

Built like the package's other class-form models: construct, ``load_state_dict``, then ``forward()`` inside
``ctx.forward_batch(batch)`` with metadata prepared by the "b200_hybrid" backend.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernel import float_ops as fo
from ..layers.base import BaseOP, OPList, StateDict
from ..layers.float_linear import FloatLinear, XieluMLP, padded_rows, take, take_f32
from ..layers.latent_attention import LatentAttention
from ..layers.recurrent import MinGRU
from ..layers.rotary_float import rotary_table
from .config import HybridLayerConfig, SefevikConfig
from .hybrid import HybridForCausalLM


class SefevikLayer(BaseOP):
    def __init__(self, config: SefevikConfig, layer: HybridLayerConfig, layer_id: int, ropes: dict, dtype: torch.dtype, device):
        hidden = config.hidden_size
        self._hidden, self._id, self._eps, self._device = hidden, layer_id, config.norm_eps, device
        if layer.type == "mingru":
            self.mix: BaseOP = MinGRU(layer.mixer, hidden, layer_id, dtype, device)
        else:
            self.mix = LatentAttention(layer.mixer, hidden, layer_id, config.norm_eps, ropes[layer.mixer.rot], dtype, device)
        self.mlp: Optional[XieluMLP] = XieluMLP(hidden, layer.mlp.ff, dtype, device) if layer.mlp is not None else None

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        self.norm1 = take_f32(state_dict, prefix + "norm1", (self._hidden,), self._device)
        self.mix.load_state_dict(state_dict, prefix=prefix + "mix.")
        if self.mlp is not None:
            self.norm2 = take_f32(state_dict, prefix + "norm2", (self._hidden,), self._device)
            self.mlp.load_state_dict(state_dict, prefix=prefix + "mlp.")
        else:
            state_dict.pop(prefix + "norm2", None)         # a gain without a sublayer has nothing to act on
        self.dwa = take_f32(state_dict, prefix + "dwa", (self._id + 2,), self._device)

    def forward(self, x_in: torch.Tensor, x: Optional[torch.Tensor], x_mid: torch.Tensor, xt: torch.Tensor, hist: torch.Tensor, md, cache,
                final_w: Optional[torch.Tensor] = None) -> None:
        """``x_in`` fp32 and ``xt`` (its copy in the model's dtype) enter; the averaged stream leaves in ``x`` (None: not
        needed) and ``xt``.  ``x_mid`` holds the stream between the sublayers; hist[:id + 1] are X_0 .. X_id."""
        dtype, planes = xt.dtype, self._id + 1
        end = dict(hist=hist, planes=planes, coef=self.dwa, hist_out=hist[planes] if planes < hist.shape[0] else None, final_w=final_w)
        if self.mlp is None:
            fo.sublayer_end(self.mix.forward(xt, md, cache), x_in, self.norm1, self._eps, x, xt, dtype, **end)
        else:
            fo.sublayer_end(self.mix.forward(xt, md, cache), x_in, self.norm1, self._eps, x_mid, xt, dtype)
            fo.sublayer_end(self.mlp.forward(xt), x_mid, self.norm2, self._eps, x, xt, dtype, **end)


class SefevikForCausalLM(HybridForCausalLM):
    def __init__(self, config: SefevikConfig, dtype: torch.dtype = torch.bfloat16, device="cuda", max_position: int = 4096):
        self._config, self._dtype, self._device = config, dtype, torch.device(device)
        fo.dtype_code(dtype)
        ropes: dict = {}
        for i in config.attention_layers:
            rot = config.layers[i].mixer.rot
            if rot not in ropes:
                ropes[rot] = rotary_table(rot, max_position, self._device)
        self.layers = OPList([SefevikLayer(config, l, i, ropes, dtype, self._device) for i, l in enumerate(config.layers)])
        self.head = FloatLinear(config.hidden_size, [config.vocab_size], ["head"], dtype, self._device)

    def load_state_dict(self, state_dict: StateDict, *, prefix: str = "", _internal: bool = False) -> None:
        c = self._config
        table = lambda name, n: take(state_dict, prefix + name, (n, c.hidden_size)).to(device=self._device, dtype=self._dtype).contiguous()
        self.embed = table("embed", c.vocab_size)
        self.bigram = table("bigram", c.bigram.buckets + 1) if c.bigram is not None else None
        for i, layer in enumerate(self.layers.op_list):
            layer.load_state_dict(state_dict, prefix=f"{prefix}l{i}.", _internal=True)
        self.final_norm = take_f32(state_dict, prefix + "final.norm", (c.hidden_size,), self._device)
        self.head.load_state_dict(state_dict, prefix=prefix)
        if not _internal and state_dict:
            raise RuntimeError(f"Unexpected keys in state_dict: {list(state_dict.keys())}")

    def forward_tokens(self, ids: torch.Tensor, md, cache, logit_rows: Optional[torch.Tensor] = None,
                       trace: Optional[List[torch.Tensor]] = None) -> Optional[torch.Tensor]:
        """fp32 logits [rows, vocab] of the token rows ``logit_rows`` (all rows when None; None for an empty selection).
        ``trace`` receives a copy of the stream that leaves every layer."""
        c, T = self._config, ids.numel()
        f32 = lambda *s: torch.empty(s, dtype=torch.float32, device=self._device)
        layers = self.layers.op_list
        hist = f32(max(len(layers), 1), T, c.hidden_size)
        xt_buf = torch.empty((T, fo.pad8(c.hidden_size)), dtype=self._dtype, device=self._device)
        xt = xt_buf[:, :c.hidden_size]
        big = c.bigram
        fo.embed_bigram(self.embed, self.bigram, ids, md.positions, md.seq_ids, md.seq_start, md.slots, cache.prev_tokens,
                        big.buckets if big else 0, big.mul_prev if big else 0, big.mul_cur if big else 0, hist[0], xt)
        x_in, x = hist[0], f32(T, c.hidden_size)
        for i, layer in enumerate(layers):
            last = i + 1 == len(layers)
            layer.forward(x_in, None if last and trace is None else x, x, xt, hist, md, cache, self.final_norm if last else None)
            x_in = x
            if trace is not None:
                trace.append(x.clone())
        if logit_rows is not None:
            if logit_rows.numel() == 0:
                return None
            xt = xt_buf.index_select(0, logit_rows)[:, :c.hidden_size]
        return self.head.forward(xt, out_f32=True)


def random_weights(config: SefevikConfig, seed: int, device="cpu", dtype: torch.dtype = torch.bfloat16) -> StateDict:
    """Seeded random weights under the checkpoint's names, scaled so that streams keep a moderate size."""
    dev = torch.device(device)
    g = torch.Generator(device=dev).manual_seed(seed)
    rnd = lambda *s: torch.randn(s, generator=g, device=dev)
    mat = lambda n, k: (rnd(n, k) * k ** -0.5).to(dtype)
    gain = lambda n: (1.0 + 0.2 * rnd(n)).to(dtype)
    W = config.hidden_size
    sd: StateDict = {"embed": rnd(config.vocab_size, W).to(dtype)}
    if config.bigram is not None:
        sd["bigram"] = (0.5 * rnd(config.bigram.buckets + 1, W)).to(dtype)
    for i, l in enumerate(config.layers):
        p, m = f"l{i}.", l.mixer
        sd[p + "norm1"] = gain(W)
        if l.type == "mingru":
            for k in ("z", "x"):
                sd[p + f"mix.{k}"], sd[p + f"mix.{k}.b"] = mat(m.width, W), rnd(m.width).to(dtype)
            sd[p + "mix.g"], sd[p + "mix.o"] = mat(m.width, W), mat(W, m.width)
        else:
            sd[p + "mix.q"] = mat(m.heads * (m.dim + m.rot_dim), W)
            if m.kv_from is None:
                sd[p + "mix.dkv"], sd[p + "mix.dkv.norm"] = mat(m.kv_rank + m.rot_dim, W), gain(m.kv_rank)
            sd[p + "mix.uk"], sd[p + "mix.uv"] = mat(m.heads * m.dim, m.kv_rank), mat(m.heads * m.vdim, m.kv_rank)
            sd[p + "mix.sink"], sd[p + "mix.o"] = rnd(m.heads).to(dtype), mat(W, m.heads * m.vdim)
        if l.mlp is not None:
            sd[p + "norm2"] = gain(W)
            sd[p + "mlp.up"], sd[p + "mlp.down"], sd[p + "mlp.act"] = mat(l.mlp.ff, W), mat(W, l.mlp.ff), (0.5 * rnd(2)).to(dtype)
        dwa = 0.3 * rnd(i + 2)
        dwa[-1] += 1.0
        sd[p + "dwa"] = dwa.to(dtype)
    sd["final.norm"], sd["head"] = gain(W), mat(config.vocab_size, W)
    return sd
