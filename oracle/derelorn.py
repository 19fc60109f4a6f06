"""Plain restatement of the Derelorn design in numpy, one function per mechanism, whole sequences at a time.

Nothing here is shared with the product path and nothing is clever: recurrences are Python loops over tokens in the order
in which their equations are written, every attention score is formed.  ``dtype`` float64 gives the oracle its own head
room; float32 shows what 32-bit rounding alone does.

Weights are a dict of arrays under the checkpoint's names ("l0.mix.q", ...), the configuration the dict that config.json
holds.
"""
from __future__ import annotations

import numpy as np

from .sefevik import rms_norm, sigmoid, silu, softplus, window_mask


# ----------------------------------------------------------------------------- short convolution
def causal_conv(x, w, bias=None):
    """Per channel: out[t] = sum_j w[:, j] x[t - (taps - 1) + j] (+ bias), zeros in front of the sequence."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1]), dtype=x.dtype), x])
    out = sum(padded[j:j + len(x)] * w[:, j] for j in range(taps))
    return out if bias is None else out + bias


# ----------------------------------------------------------------------------- matrix memory with exponential gates
def mlstm_scan(q, k, v, i, f):
    """q, k [T, H, dim], v [T, H, vdim], log gates i, f [T, H]; read-outs [T, H, vdim].  The exponentials are kept in
    range by a running maximum that starts at 0."""
    T, H, dim = q.shape
    S, n, m = np.zeros((H, dim, v.shape[2]), q.dtype), np.zeros((H, dim), q.dtype), np.zeros(H, q.dtype)
    out = np.empty(v.shape, q.dtype)
    for t in range(T):
        new = np.maximum(f[t] + m, i[t])
        keep, write = np.exp(f[t] + m - new), np.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = new
        den = np.maximum(np.abs(np.sum(n * q[t], axis=1)), np.exp(-m)) + 1e-6
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


def mlstm(h, mix, w, pre, eps):
    T, H, dim, vdim, cap = len(h), mix["heads"], mix["dim"], mix["vdim"], mix["gate_cap"]
    soft_cap = lambda z: cap * np.tanh(z / cap)
    q = (h @ w[pre + "q"].T * dim ** -0.5).reshape(T, H, dim)
    k = (h @ w[pre + "k"].T).reshape(T, H, dim)
    v = (h @ w[pre + "v"].T).reshape(T, H, vdim)
    i = soft_cap(h @ w[pre + "i"].T + w[pre + "i.b"])
    f = -softplus(-soft_cap(h @ w[pre + "f"].T + w[pre + "f.b"]))
    o = rms_norm(mlstm_scan(q, k, v, i, f), 1.0, eps).reshape(T, H * vdim)
    return (o * w[pre + "norm"] * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ----------------------------------------------------------------------------- gated delta rule
def delta_scan(q, k, v, beta, g):
    """q, k [T, H, dim] unit vectors (q scaled), v [T, H, vdim], write strengths beta and decays g [T, H]."""
    T, H, dim = q.shape
    S, out = np.zeros((H, dim, v.shape[2]), q.dtype), np.empty(v.shape, q.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta(h, mix, w, pre, eps):
    T, H, G, dim, vdim = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    conv = lambda name: silu(causal_conv(h @ w[pre + name].T, w[pre + name + ".conv"]))
    share = np.arange(H) // (H // G)                      # the q / k head of every head
    q = unit(conv("q").reshape(T, G, dim))[:, share] * dim ** -0.5
    k = unit(conv("k").reshape(T, G, dim))[:, share]
    v = conv("v").reshape(T, H, vdim)
    beta = sigmoid(h @ w[pre + "b"].T)
    g = np.exp(-np.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o = rms_norm(delta_scan(q, k, v, beta, g), w[pre + "norm"], eps).reshape(T, H * vdim)
    return (o * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ----------------------------------------------------------------------------- state-space duality (Mamba-2)
def ssd_scan(x, B, C, dt, decay, D):
    """x [T, H, vdim], B, C [T, H, N] (groups already spread over the heads), dt, decay [T, H], D [H]."""
    T, H, vdim = x.shape
    S, out = np.zeros((H, B.shape[2], vdim), x.dtype), np.empty(x.shape, x.dtype)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = np.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return out


def mamba2(h, mix, w, pre, eps):
    T, H, vdim, N, G = len(h), mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    inner = H * vdim
    z, xbc, dt = np.split(h @ w[pre + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    share = np.arange(H) // (H // G)
    dt = softplus(dt + w[pre + "dt_bias"])
    decay = np.exp(-np.exp(w[pre + "A_log"]) * dt)
    y = ssd_scan(x.reshape(T, H, vdim), B.reshape(T, G, N)[:, share], C.reshape(T, G, N)[:, share], dt, decay, w[pre + "D"])
    y = (y.reshape(T, inner) * silu(z)).reshape(T, mix["norm_groups"], -1)
    return (rms_norm(y, 1.0, eps).reshape(T, inner) * w[pre + "norm"]) @ w[pre + "o"].T


# ----------------------------------------------------------------------------- windowed attention with shared key heads
def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def grouped_attention(q, k, v, window, scale):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    per, mask = H // k.shape[1], window_mask(T, window)
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for hd in range(H):
        s = np.where(mask, (q[:, hd] @ k[:, hd // per].T) * scale, -np.inf)
        out[:, hd] = softmax(s) @ v[:, hd // per]
    return out


def attention(h, mix, w, pre, eps):
    T, H, G = len(h), mix["heads"], mix["kv_heads"]
    q = rms_norm(h @ w[pre + "q"].T, w[pre + "q.norm"], eps).reshape(T, H, mix["dim"])
    k = rms_norm(h @ w[pre + "k"].T, w[pre + "k.norm"], eps).reshape(T, G, mix["dim"])
    v = (h @ w[pre + "v"].T).reshape(T, G, mix["vdim"])
    o = grouped_attention(q, k, v, (mix.get("mask") or {}).get("size"), mix["scale"])
    return o.reshape(T, -1) @ w[pre + "o"].T


def parallel(h, mix, w, pre, eps):
    left = attention(h, mix["left"], w, pre + "left.", eps)
    right = mamba2(h, mix["right"], w, pre + "right.", eps)
    return 0.5 * (rms_norm(left, w[pre + "left.out"], eps) + rms_norm(right, w[pre + "right.out"], eps))


# ----------------------------------------------------------------------------- feed-forward and model
def gated_mlp(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


MIXERS = {"mlstm": mlstm, "delta": delta, "parallel": parallel}


def schedule(cfg):
    """(layer, pass that begins with it or None) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    body = range(loop["start"], loop["stop"])
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in body]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(tokens, cfg, weights, dtype=np.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) receives the stream that leaves every run of a layer."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    for i, begins in schedule(cfg):
        layer, pre = cfg["layers"][i], f"l{i}."
        if begins is not None:
            x = x + w["loop.step"][begins]
        y = MIXERS[layer["type"]](rms_norm(x, w[pre + "norm1"], eps), layer["mixer"], w, pre + "mix.", eps)
        x = x + rms_norm(y, w[pre + "norm1b"], eps)
        if layer.get("mlp"):
            y = gated_mlp(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.")
            x = x + rms_norm(y, w[pre + "norm2b"], eps)
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
