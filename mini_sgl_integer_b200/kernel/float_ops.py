"""Tensor-level wrappers of the floating-point kernels (``include/b200float.h``).

Activations between kernels are rows of one dtype (bfloat16 or float32) whose pitch is a multiple of 8 values
(``rows``).  A linear whose consumer is one of these kernels may stay a stack of fp32 partial sums [parts, rows, n]
(``linear_parts``); the consumer adds the parts in order.  Everything runs on the current stream and raises when a
tensor is not on a CUDA device or an argument is rejected.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._lib import call, ptr, query, require_cuda, stream

ACT_NONE, ACT_XIELU = 0, 1
_CODES = {torch.float32: 0, torch.bfloat16: 1}


def dtype_code(dtype: torch.dtype) -> int:
    if dtype not in _CODES:
        raise TypeError(f"the floating-point kernels take float32 or bfloat16, got {dtype}")
    return _CODES[dtype]


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def rows(count: int, n: int, dtype: torch.dtype, device) -> torch.Tensor:
    """Uninitialised [count, n] whose row pitch is a multiple of 8 values."""
    return torch.empty((count, pad8(n)), dtype=dtype, device=device)[:, :n]


def _check_rows(name: str, t: torch.Tensor, dtype: torch.dtype, n: Optional[int] = None) -> None:
    if t.dtype != dtype:
        raise TypeError(f"{name} must be {dtype}, got {t.dtype}")
    if t.ndim != 2 or (t.shape[1] > 1 and t.stride(1) != 1) or (n is not None and t.shape[1] != n):
        raise ValueError(f"{name} must be rows{'' if n is None else f' of {n} values'}, got {tuple(t.shape)} with strides {t.stride()}")
    require_cuda(t)


def _check_parts(name: str, t: torch.Tensor, n: int) -> None:
    if t.dtype != torch.float32 or t.ndim != 3 or t.shape[2] != n or not t.is_contiguous():
        raise ValueError(f"{name} must be contiguous fp32 [parts, rows, {n}], got {t.dtype} {tuple(t.shape)}")
    require_cuda(t)


def _check_vec(name: str, t: torch.Tensor, n: int) -> None:
    if t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous():
        raise ValueError(f"{name} must be {n} contiguous fp32 values, got {t.dtype} {tuple(t.shape)}")
    require_cuda(t)


# ----------------------------------------------------------------------------- linears
def linear(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, out_f32: bool = False, act: int = ACT_NONE,
           act_a: float = 0.0, act_b: float = 0.0) -> torch.Tensor:
    """act(x w^T) for rows x [T, k] and weight rows w [n, k]."""
    _check_rows("x", x, x.dtype)
    _check_rows("w", w, x.dtype, x.shape[1])
    T, k = x.shape
    n = w.shape[0]
    if out is None:
        out = rows(T, n, torch.float32 if out_f32 else x.dtype, x.device)
    out_f32 = out.dtype == torch.float32
    call("b200f_gemm", ptr(x), ptr(w), ptr(out), dtype_code(x.dtype), int(out_f32), T, n, k, 1, _pitch(x), 0, _pitch(w), 0,
         _pitch(out), 0, 1, 0, act, act_a, act_b, stream())
    return out


def linear_parts(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x w^T as fp32 partial sums [parts, T, n]; several parts at decode sizes where the weight alone cannot occupy the GPU."""
    _check_rows("x", x, x.dtype)
    _check_rows("w", w, x.dtype, x.shape[1])
    T, k = x.shape
    n, code = w.shape[0], dtype_code(x.dtype)
    parts = query("b200f_gemm_splits", T, n, k, 1, code)
    out = torch.empty((parts, T, n), dtype=torch.float32, device=x.device)
    call("b200f_gemm", ptr(x), ptr(w), ptr(out), code, 1, T, n, k, 1, _pitch(x), 0, _pitch(w), 0, n, 0, parts, T * n, ACT_NONE,
         0.0, 0.0, stream())
    return out


def _pitch(t: torch.Tensor) -> int:
    return t.stride(0) if t.shape[0] > 1 else max(t.stride(0), t.shape[1])


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """out[:, h] = x[:, h] w[h]^T for every head: x [T, H, k], w [H, n, k], out [T, H, n] views of one dtype."""
    T, H, k = x.shape
    n = w.shape[1]
    if x.dtype != w.dtype or out.dtype != x.dtype or w.shape != (H, n, k) or out.shape != (T, H, n):
        raise ValueError(f"head_linear: x {tuple(x.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    if x.stride(2) != 1 or w.stride(2) != 1 or out.stride(2) != 1:
        raise ValueError("head_linear: rows must be contiguous")
    require_cuda(x, w, out)
    call("b200f_gemm", ptr(x), ptr(w), ptr(out), dtype_code(x.dtype), int(out.dtype == torch.float32), T, n, k, H, x.stride(0), x.stride(1),
         w.stride(1), w.stride(0), out.stride(0), out.stride(1), 1, 0, ACT_NONE, 0.0, 0.0, stream())


def check_status() -> None:
    """Raises if a bounded wait inside a linear or the attention kernel has expired since the last check.  Synchronises
    with the device."""
    for name, what in (("b200f_gemm_status", "a bf16 linear"), ("b200f_latent_attn_status", "the latent attention kernel")):
        st = ctypes.c_int(0)
        call(name, ctypes.byref(st), 1)
        if st.value:
            raise RuntimeError(f"a wait inside {what} expired (code {st.value}: 1 loader, 2 MMA issuer, 3 epilogue, 4 accumulator "
                               "hand-back, 5 copying warp, 6 consumer); the step's results are not valid")


# ----------------------------------------------------------------------------- ends of a model
def embed_bigram(table, bigram, ids, positions, seq_ids, seq_start, slots, prev_tokens, buckets: int, mul_prev: int, mul_cur: int,
                 out: torch.Tensor, out_t: Optional[torch.Tensor]) -> None:
    """Embedding row (+ bigram row unless ``bigram`` is None) of every token into fp32 ``out`` [T, width] and rows ``out_t``."""
    require_cuda(table, bigram, ids, out, out_t)
    T, width = out.shape
    call("b200f_embed_bigram", ptr(table), ptr(bigram), ptr(ids), ptr(positions), ptr(seq_ids), ptr(seq_start), ptr(slots), ptr(prev_tokens),
         ptr(out), ptr(out_t), dtype_code(table.dtype), T, width, table.shape[0], buckets, mul_prev, mul_cur,
         0 if out_t is None else _pitch(out_t), stream())


def argmax_f32(logits: torch.Tensor) -> torch.Tensor:
    """Row-wise arg-max of fp32 logits, the lowest index on ties."""
    _check_rows("logits", logits, torch.float32)
    idx = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    call("b200f_argmax", ptr(logits), logits.shape[0], logits.shape[1], _pitch(logits), ptr(idx), stream())
    return idx


# ----------------------------------------------------------------------------- rows
def sublayer_end(y: torch.Tensor, x_in: torch.Tensor, norm_w: torch.Tensor, eps: float, x_out: Optional[torch.Tensor],
                 x_out_t: Optional[torch.Tensor], dtype: torch.dtype, hist: Optional[torch.Tensor] = None, planes: int = 0,
                 coef: Optional[torch.Tensor] = None, hist_out: Optional[torch.Tensor] = None,
                 final_w: Optional[torch.Tensor] = None) -> None:
    """r = x_in + rmsnorm(y) * norm_w; with ``coef`` then the depth average over hist[:planes] and r (r kept in
    ``hist_out``), with ``final_w`` then that norm on the way to ``x_out_t``.  See b200f_sublayer_end."""
    T, width = x_in.shape
    _check_parts("y", y, width)
    _check_vec("norm_w", norm_w, width)
    for t in (x_in, x_out, hist_out):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous() or t.shape != (T, width)):
            raise ValueError("sublayer_end: streams must be contiguous fp32 [rows, width]")
    if x_out_t is not None:
        _check_rows("x_out_t", x_out_t, dtype, width)
    if coef is not None:
        _check_vec("coef", coef, planes + 1)
        if hist is None or hist.dtype != torch.float32 or not hist.is_contiguous() or hist.shape[0] < planes or hist.shape[1:] != (T, width):
            raise ValueError("sublayer_end: hist must be contiguous fp32 [planes, rows, width]")
    call("b200f_sublayer_end", ptr(y), y.shape[0], T * width, ptr(x_in), ptr(norm_w), ptr(x_out), ptr(x_out_t), ptr(hist), planes, T * width,
         ptr(coef), ptr(hist_out), ptr(final_w), dtype_code(dtype), T, width, 0 if x_out_t is None else _pitch(x_out_t), float(eps), stream())


def xielu(y: torch.Tensor, out: torch.Tensor, act_a: float, act_b: float) -> None:
    _check_parts("y", y, out.shape[1])
    call("b200f_xielu", ptr(y), y.shape[0], y.shape[1] * y.shape[2], ptr(out), dtype_code(out.dtype), y.shape[1], y.shape[2], _pitch(out),
         act_a, act_b, stream())


# ----------------------------------------------------------------------------- mixers
def mingru(zug: torch.Tensor, bias_z: torch.Tensor, bias_u: torch.Tensor, state: torch.Tensor, slots, positions, seq_start,
           batch: int, out: torch.Tensor) -> None:
    """Gated recurrence over pre-activations z | u | g [parts, T, 3 width]; ``state`` fp32 [slots, width] is updated."""
    T, width = out.shape
    _check_parts("zug", zug, 3 * width)
    _check_vec("bias_z", bias_z, width)
    _check_vec("bias_u", bias_u, width)
    if state.dtype != torch.float32 or state.ndim != 2 or state.shape[1] != width or not state.is_contiguous():
        raise ValueError(f"state must be contiguous fp32 [slots, {width}]")
    call("b200f_mingru", ptr(zug), zug.shape[0], zug.shape[1] * zug.shape[2], ptr(bias_z), ptr(bias_u), ptr(state), ptr(slots), ptr(positions),
         ptr(seq_start), ptr(out), dtype_code(out.dtype), T, batch, width, _pitch(out), stream())


def latent_prepare(qd: torch.Tensor, positions, out_loc, rope: Optional[torch.Tensor], dkv_norm: Optional[torch.Tensor], eps: float,
                   qn: torch.Tensor, q_lat: torch.Tensor, cache: Optional[torch.Tensor], heads: int, dim: int, rot_dim: int,
                   kv_rank: int) -> None:
    """Splits and rotates the projections of latent attention; see b200f_latent_prepare.  qn [T, heads, >= dim],
    q_lat [T, heads, pitch], cache [pages, 16, pitch] (with ``dkv_norm``)."""
    parts, T, n = qd.shape
    _check_parts("qd", qd, heads * (dim + rot_dim) + (0 if dkv_norm is None else kv_rank + rot_dim))
    if dkv_norm is not None:
        _check_vec("dkv_norm", dkv_norm, kv_rank)
    require_cuda(qn, q_lat, cache)
    pitch = q_lat.shape[2]
    call("b200f_latent_prepare", ptr(qd), parts, T * n, n, ptr(positions), ptr(out_loc), ptr(rope), 0 if rope is None else rope.shape[1],
         1 if rope is None else rope.shape[0], ptr(dkv_norm), float(eps), ptr(qn), ptr(q_lat), ptr(cache), dtype_code(q_lat.dtype), T, heads,
         dim, rot_dim, kv_rank, dim + rot_dim, qn.shape[2], pitch, 0 if cache is None else cache.shape[0] * cache.shape[1], stream())


def latent_attention(q_lat: torch.Tensor, cache: torch.Tensor, page_table: torch.Tensor, kv_lens, seq_start, sink: torch.Tensor,
                     out: torch.Tensor, kv_rank: int, rot_dim: int, window: int, scale: float, max_q: int, max_kv: int,
                     key_splits: int = 0, simple: bool = False) -> None:
    """Attention of queries in the latent space over the paged cache; see b200f_latent_attn.  out [T, heads, >= kv_rank].
    ``key_splits`` 0 lets the library choose over how many CTAs a query tile's keys are spread."""
    T, heads, pitch = q_lat.shape
    if cache.dtype != q_lat.dtype or cache.shape[2] != pitch or out.dtype != q_lat.dtype or not (q_lat.is_contiguous() and cache.is_contiguous() and out.is_contiguous()):
        raise ValueError("latent_attention: q_lat, cache and out must be contiguous and of one dtype, q_lat and cache of one pitch")
    _check_vec("sink", sink, heads)
    require_cuda(q_lat, cache, page_table, kv_lens, out)
    code, batch = dtype_code(q_lat.dtype), kv_lens.numel()
    if simple:
        key_splits = 1
    elif key_splits <= 0:
        key_splits = query("b200f_latent_attn_splits", T, batch, max_q, max_kv, heads, kv_rank, rot_dim, window, code)
    floats = query("b200f_latent_attn_ws_floats", T, heads, kv_rank, key_splits)
    ws = torch.empty(floats, dtype=torch.float32, device=q_lat.device) if floats else None
    call("b200f_latent_attn", ptr(q_lat), ptr(cache), ptr(page_table), page_table.stride(0), ptr(kv_lens), ptr(seq_start), ptr(sink), ptr(out),
         code, T, batch, max_q, heads, kv_rank, rot_dim, pitch, out.shape[2], window, float(scale), key_splits, ptr(ws), int(simple), stream())
