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

ACT_NONE, ACT_XIELU, ACT_GATED_SILU = 0, 1, 2
MEMORY_EXP, MEMORY_SSD, MEMORY_DELTA = 0, 1, 2
GATE_SILU_BEFORE, GATE_SIGMOID_AFTER, GATE_SILU_AFTER = 0, 1, 2
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
    """act(x w^T) for rows x [T, k] and weight rows w [n, k]; with ACT_GATED_SILU (bf16) the weight rows alternate, 16 gates
    and 16 values, and the result has n / 2 columns."""
    _check_rows("x", x, x.dtype)
    _check_rows("w", w, x.dtype, x.shape[1])
    T, k = x.shape
    n = w.shape[0]
    if out is None:
        out = rows(T, n // 2 if act == ACT_GATED_SILU else n, torch.float32 if out_f32 else x.dtype, x.device)
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
    """Raises if a bounded wait inside a linear, the latent attention kernel or the chunked scan has expired since the last
    check.  Synchronises with the device."""
    for name, what in (("b200f_gemm_status", "a bf16 linear"), ("b200f_latent_attn_status", "the latent attention kernel"),
                       ("b200f_memory_scan_status", "the scan of a matrix memory")):
        st = ctypes.c_int(0)
        call(name, ctypes.byref(st), 1)
        if st.value:
            raise RuntimeError(f"a wait inside {what} expired (code {st.value}: 1 loader, 2 MMA issuer, 3 epilogue, 4 accumulator "
                               "hand-back, 5 copying warp, 6 consumer, 7 chunk); the step's results are not valid")


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
def sublayer_end(y: Optional[torch.Tensor], x_in: Optional[torch.Tensor], norm_w: Optional[torch.Tensor], eps: float,
                 x_out: Optional[torch.Tensor], x_out_t: Optional[torch.Tensor], dtype: torch.dtype, hist: Optional[torch.Tensor] = None,
                 planes: int = 0, coef: Optional[torch.Tensor] = None, hist_out: Optional[torch.Tensor] = None,
                 final_w: Optional[torch.Tensor] = None, mean_with: Optional[tuple] = None, add: Optional[torch.Tensor] = None) -> None:
    """r = x_in + rmsnorm(y) * norm_w (``x_in`` None: zero; ``y`` None: r = x_in), plus the vector ``add``; with ``coef``
    then the depth average over hist[:planes] and r (r kept in ``hist_out``), with ``final_w`` then that norm on the way to
    ``x_out_t``.  ``mean_with`` (w1, y2, w2): the mean of rmsnorm(y) * w1 and rmsnorm(y2) * w2 takes the place of y.  x_in and
    x_out may be the same tensor.  See b200f_sublayer_end."""
    T, width = (y.shape[1:] if x_in is None else x_in.shape)
    if y is not None:
        _check_parts("y", y, width)
        _check_vec("norm_w", norm_w, width)
    w1, y2, w2 = mean_with or (None, None, None)
    if mean_with is not None:
        _check_parts("y2", y2, width)
        _check_vec("w1", w1, width)
        _check_vec("w2", w2, width)
    for name, t in (("add", add), ("final_w", final_w)):
        if t is not None:
            _check_vec(name, t, width)
    for t in (x_in, x_out, hist_out):
        if t is not None and (t.dtype != torch.float32 or not t.is_contiguous() or t.shape != (T, width)):
            raise ValueError("sublayer_end: streams must be contiguous fp32 [rows, width]")
    if x_out_t is not None:
        _check_rows("x_out_t", x_out_t, dtype, width)
    if coef is not None:
        _check_vec("coef", coef, planes + 1)
        if hist is None or hist.dtype != torch.float32 or not hist.is_contiguous() or hist.shape[0] < planes or hist.shape[1:] != (T, width):
            raise ValueError("sublayer_end: hist must be contiguous fp32 [planes, rows, width]")
    call("b200f_sublayer_end", ptr(y), 1 if y is None else y.shape[0], T * width, ptr(y2), 1 if y2 is None else y2.shape[0], T * width, ptr(w1),
         ptr(w2), ptr(x_in), ptr(norm_w), ptr(add), ptr(x_out), ptr(x_out_t), ptr(hist), planes, T * width, ptr(coef), ptr(hist_out), ptr(final_w),
         dtype_code(dtype), T, width, 0 if x_out_t is None else _pitch(x_out_t), float(eps), stream())


def gated_silu(y: torch.Tensor, out: torch.Tensor) -> None:
    """silu(gate) * value over parts [parts, T, n] whose columns alternate, 16 gates and 16 values; out rows [T, <= n / 2]."""
    _check_parts("y", y, y.shape[2])
    call("b200f_gated_silu", ptr(y), y.shape[0], y.shape[1] * y.shape[2], y.shape[2], ptr(out), dtype_code(out.dtype), y.shape[1], out.shape[1],
         _pitch(out), stream())


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


def memory_prepare(y: torch.Tensor, col0: int, segments, conv_w: Optional[torch.Tensor], conv_b: Optional[torch.Tensor],
                   conv_state: Optional[torch.Tensor], slots, positions, seq_start, seq_ids, out: torch.Tensor, kind: int, heads: int,
                   gate_cols, gate_a: torch.Tensor, gate_b: torch.Tensor, gates: torch.Tensor, cap: float = 0.0,
                   norm_state: Optional[torch.Tensor] = None) -> None:
    """Between the projections of a matrix recurrence and its scan; see b200f_memory_prepare.  ``segments``: three pairs
    (columns, head size); out rows of padded heads; gates fp32 [T, heads, 4]."""
    parts, T, n = y.shape
    _check_parts("y", y, n)
    width, padded = sum(w for w, _ in segments), sum(w // h * pad8(h) for w, h in segments)
    _check_rows("out", out, out.dtype, padded)
    _check_vec("gates", gates, T * heads * 4)
    _check_vec("gate_a", gate_a, heads)
    _check_vec("gate_b", gate_b, heads)
    taps = 0
    if conv_w is not None:
        taps = conv_w.shape[1]
        _check_vec("conv_w", conv_w, width * taps)
        if conv_b is not None:
            _check_vec("conv_b", conv_b, width)
        if taps > 1 and (conv_state.dtype != torch.float32 or conv_state.shape[1:] != (taps - 1, width) or not conv_state.is_contiguous()):
            raise ValueError(f"conv_state must be contiguous fp32 [slots, {taps - 1}, {width}]")
    if kind == MEMORY_EXP and (norm_state.dtype != torch.float32 or norm_state.shape[1] != heads or not norm_state.is_contiguous()):
        raise ValueError(f"norm_state must be contiguous fp32 [slots, {heads}, dim + 1]")
    seg = (ctypes.c_int32 * 6)(*[v for s in segments for v in s])
    call("b200f_memory_prepare", ptr(y), parts, T * n, n, col0, ctypes.cast(seg, ctypes.c_void_p), ptr(conv_w), ptr(conv_b), taps,
         ptr(conv_state) if taps > 1 else None, ptr(slots), ptr(positions), ptr(seq_start), ptr(seq_ids), ptr(out), _pitch(out), dtype_code(out.dtype),
         kind, heads, gate_cols[0], gate_cols[1], ptr(gate_a), ptr(gate_b), float(cap), ptr(gates), ptr(norm_state),
         0 if norm_state is None else norm_state.shape[2] - 1, T, slots.numel(), stream())


def memory_scan(rows_: torch.Tensor, offsets, qk_heads: int, heads: int, dim: int, vdim: int, kind: int, gates: torch.Tensor, q_scale: float,
                skip: Optional[torch.Tensor], state: torch.Tensor, norm_state: Optional[torch.Tensor], slots, positions, seq_start,
                out: torch.Tensor, den: Optional[torch.Tensor], max_q: int, simple: bool = False) -> None:
    """Read-outs of a matrix recurrence; ``state`` fp32 [slots, heads, dim, round8(vdim)] is updated; see b200f_memory_scan.
    ``offsets``: columns of the first q, k and v head; out fp32 [T, heads * vdim], den fp32 [T, heads].  ``max_q``: most new
    tokens of a sequence; ``simple``: token by token also where chunks on the tensor cores would do."""
    T = rows_.shape[0]
    _check_rows("rows", rows_, rows_.dtype)
    _check_vec("gates", gates, T * heads * 4)
    _check_vec("out", out, T * heads * vdim)
    if state.dtype != torch.float32 or state.shape[1:] != (heads, dim, pad8(vdim)) or not state.is_contiguous():
        raise ValueError(f"state must be contiguous fp32 [slots, {heads}, {dim}, {pad8(vdim)}]")
    if skip is not None:
        _check_vec("skip", skip, heads)
    if kind == MEMORY_EXP:
        _check_vec("den", den, T * heads)
        if norm_state.shape[1:] != (heads, dim + 1) or not norm_state.is_contiguous():
            raise ValueError(f"norm_state must be contiguous fp32 [slots, {heads}, {dim + 1}]")
    need = 0 if simple or seq_start is None else query("b200f_memory_scan_ws_bytes", T, slots.numel(), max_q, heads, dim, vdim, kind, dtype_code(rows_.dtype))
    ws = torch.empty(need, dtype=torch.uint8, device=rows_.device) if need else None
    call("b200f_memory_scan", ptr(rows_), dtype_code(rows_.dtype), _pitch(rows_), *offsets, qk_heads, heads, dim, vdim, kind, ptr(gates),
         float(q_scale), ptr(skip), ptr(state), ptr(norm_state), ptr(slots), ptr(positions), ptr(seq_start), ptr(out), ptr(den), T, slots.numel(),
         max_q, ptr(ws), int(simple), stream())


def memory_output(o: torch.Tensor, den: Optional[torch.Tensor], heads: int, vdim: int, group: int, y: torch.Tensor, gate_col: int, gate: int,
                  norm_w: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """Read-outs [T, heads * vdim] normed in groups, with the gate in column ``gate_col`` of y; see b200f_memory_output."""
    T, n = out.shape
    _check_vec("o", o, T * n)
    _check_parts("y", y, y.shape[2])
    _check_rows("out", out, out.dtype, heads * vdim)
    _check_vec("norm_w", norm_w, norm_w.numel())
    if den is not None:
        _check_vec("den", den, T * heads)
    call("b200f_memory_output", ptr(o), ptr(den), heads, vdim, group, ptr(y), y.shape[0], y.shape[1] * y.shape[2], y.shape[2], gate_col, gate,
         ptr(norm_w), norm_w.numel(), float(eps), ptr(out), _pitch(out), dtype_code(out.dtype), T, stream())


def grouped_prepare(y: torch.Tensor, cols, q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor], eps: float, out_loc, q: torch.Tensor,
                    k_cache: torch.Tensor, v_cache: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int) -> None:
    """Norms of q and k and the cache store of grouped attention; see b200f_grouped_prepare.  q [T, heads, pad8(dim)], caches
    [pages, 16, kv_heads * pad8(size)]."""
    parts, T, n = y.shape
    _check_parts("y", y, n)
    for name, w, k in (("q_norm", q_norm, heads * dim), ("k_norm", k_norm, kv_heads * dim)):
        if w is not None:
            _check_vec(name, w, k)
    dp, vp = pad8(dim), pad8(vdim)
    if q.shape != (T, heads, dp) or k_cache.shape[2] != kv_heads * dp or v_cache.shape[2] != kv_heads * vp or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
        raise ValueError("grouped_prepare: q or the caches have other sizes or types")
    require_cuda(q, k_cache, v_cache)
    call("b200f_grouped_prepare", ptr(y), parts, T * n, n, cols[0], cols[1], cols[2], ptr(q_norm), ptr(k_norm), float(eps), ptr(out_loc), ptr(q),
         ptr(k_cache), ptr(v_cache), dtype_code(q.dtype), T, heads, kv_heads, dim, vdim, dp, vp, k_cache.shape[0] * k_cache.shape[1], stream())


def grouped_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, page_table: torch.Tensor, kv_lens, seq_start,
                      out: torch.Tensor, kv_heads: int, dim: int, vdim: int, window: int, scale: float, max_q: int, max_kv: int,
                      key_splits: int = 0, simple: bool = False) -> None:
    """Attention over paged keys and values; see b200f_grouped_attn.  out rows [T, heads * vdim].  ``key_splits`` 0 lets the
    library choose over how many CTAs a decode row's keys are spread."""
    T, heads, dp = q.shape
    vp = v_cache.shape[2] // kv_heads
    if k_cache.dtype != q.dtype or v_cache.dtype != q.dtype or k_cache.shape[2] != kv_heads * dp or not (q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise ValueError("grouped_attention: q and the caches must be contiguous and of one dtype and pitch")
    _check_rows("out", out, q.dtype, heads * vdim)
    require_cuda(q, k_cache, v_cache, page_table, kv_lens)
    code, batch = dtype_code(q.dtype), kv_lens.numel()
    if simple:
        key_splits = 1
    elif key_splits <= 0:
        key_splits = query("b200f_grouped_attn_splits", T, batch, max_q, max_kv, heads, kv_heads, dim, vdim, window, code)
    floats = query("b200f_grouped_attn_ws_floats", T, heads, vdim, key_splits)
    ws = torch.empty(floats, dtype=torch.float32, device=q.device) if floats else None
    call("b200f_grouped_attn", ptr(q), ptr(k_cache), ptr(v_cache), ptr(page_table), page_table.stride(0), ptr(kv_lens), ptr(seq_start), ptr(out),
         code, T, batch, max_q, heads, kv_heads, dim, vdim, dp, vp, _pitch(out), window, float(scale), key_splits, ptr(ws), int(simple), stream())
