"""Plain restatement of the Sefevik design in numpy, one function per mechanism, whole sequences at a time.

Nothing here is shared with the product path and nothing is clever: every attention score is formed, the recurrence
is a Python loop over tokens, the keys are expanded per head instead of attending in the latent space.  ``dtype``
float64 gives the oracle its own head room; float32 shows what 32-bit rounding alone does.

Weights are a dict of arrays under the checkpoint's names ("l0.mix.z", ...), the configuration the dict that
config.json holds.
"""
from __future__ import annotations

import math

import numpy as np


# ----------------------------------------------------------------------------- elementwise pieces
def sigmoid(v):
    e = np.exp(-np.abs(v))
    return np.where(v >= 0, 1 / (1 + e), e / (1 + e))


def softplus(v):
    return np.logaddexp(0.0, v)


def silu(v):
    return v * sigmoid(v)


def rms_norm(x, w, eps):
    """Root-mean-square norm over the last axis, eps under the root, gain w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def xielu(z, p, q):
    """Quadratic branch for positive inputs, exponential branch for the others; both have slope 1/2 at zero."""
    pos = softplus(p) * z * z + 0.5 * z
    zn = np.minimum(z, 0.0)
    neg = (0.5 + softplus(q)) * (np.expm1(zn) - zn) + 0.5 * z
    return np.where(z > 0, pos, neg)


# ----------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for each token of a sequence; the first token takes the extra last row."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return np.asarray(rows, dtype=np.int64)


def embed(tokens, cfg, w):
    x = w["embed"][np.asarray(tokens)]
    big = cfg.get("embedding", {}).get("bigram")
    if big:
        x = x + w["bigram"][bigram_rows(tokens, big["buckets"], big["mul_prev"], big["mul_cur"])]
    return x


# ----------------------------------------------------------------------------- depth average
def depth_average(history, coef):
    """Weighted sum of the embedding output and every layer result so far."""
    out = np.zeros_like(history[0])
    for c, h in zip(coef, history):
        out = out + c * h
    return out


# ----------------------------------------------------------------------------- gated recurrence
def mingru_scan(z_pre, u_pre, state=None):
    """S_t = (1 - z_t) S_(t-1) + z_t cand_t for pre-activations [T, width]; returns all states [T, width]."""
    s = np.zeros(z_pre.shape[1], dtype=z_pre.dtype) if state is None else state
    out = np.empty_like(z_pre)
    for t in range(z_pre.shape[0]):
        z = sigmoid(z_pre[t])
        cand = np.where(u_pre[t] >= 0, u_pre[t] + 0.5, sigmoid(u_pre[t]))
        s = (1 - z) * s + z * cand
        out[t] = s
    return out


def mingru(h, w, pre):
    z = h @ w[pre + "z"].T + w[pre + "z.b"]
    u = h @ w[pre + "x"].T + w[pre + "x.b"]
    s = mingru_scan(z, u)
    return (s * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ----------------------------------------------------------------------------- rotary positions
def rotary_frequencies(rot):
    """(frequencies [dims / 2], factor on cos and sin), float64."""
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(where(sc["fast"])), 0)
    hi = min(math.ceil(where(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """Rotates the first rot.dims entries of the last axis of x [T, ..., n]; entry i pairs with i + dims / 2."""
    f, m = rotary_frequencies(rot)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (len(f),)
    c, s = (np.cos(ang) * m).reshape(shape), (np.sin(ang) * m).reshape(shape)
    half = len(f)
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return np.concatenate([u * c - v * s, v * c + u * s, rest], axis=-1).astype(x.dtype)


# ----------------------------------------------------------------------------- latent attention
def latent_keys(h, mix, w, pre, eps):
    """(latent [T, kv_rank], rotated shared key part [T, rot_dim])."""
    d = h @ w[pre + "dkv"].T
    c = rms_norm(d[:, :mix["kv_rank"]], w[pre + "dkv.norm"], eps)
    kr = d[:, mix["kv_rank"]:]
    if mix.get("rot"):
        kr = rotate(kr, np.arange(len(h)), mix["rot"])
    return c, kr


def window_mask(n, size):
    """Causal band matrix: row i holds the last `size` keys up to i (every key up to i when size is None)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    ok = j <= i
    return ok if size is None else ok & (i - j < size)


def sink_softmax(scores, sink):
    """Softmax of [..., keys] whose denominator has one more term, exp(sink)."""
    m = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def latent_attention_heads(q, c, kr, mix, w, pre):
    """Attention outputs [T, heads, vdim] of projected, rotated queries q [T, heads, dim + rot_dim]."""
    H, dim, vdim = mix["heads"], mix["dim"], mix["vdim"]
    T = len(q)
    k = (c @ w[pre + "uk"].T).reshape(T, H, dim)
    v = (c @ w[pre + "uv"].T).reshape(T, H, vdim)
    mask = window_mask(T, (mix.get("mask") or {}).get("size"))
    out = np.empty((T, H, vdim), dtype=q.dtype)
    for hd in range(H):
        s = (q[:, hd, :dim] @ k[:, hd].T + q[:, hd, dim:] @ kr.T) * mix["scale"]
        s = np.where(mask, s, -np.inf)
        out[:, hd] = sink_softmax(s, w[pre + "sink"][hd]) @ v[:, hd]
    return out


def latent_attention(h, mix, w, pre, eps, shared):
    """``shared``: (latent, key part) of the layer that kv_from names, or None.  Returns (output, its own pair)."""
    T, H = len(h), mix["heads"]
    q = (h @ w[pre + "q"].T).reshape(T, H, mix["dim"] + mix["rot_dim"])
    if mix.get("rot"):
        q = np.concatenate([q[..., :mix["dim"]], rotate(q[..., mix["dim"]:], np.arange(T), mix["rot"])], axis=-1)
    c, kr = shared if shared is not None else latent_keys(h, mix, w, pre, eps)
    o = latent_attention_heads(q, c, kr, mix, w, pre)
    return o.reshape(T, -1) @ w[pre + "o"].T, (c, kr)


# ----------------------------------------------------------------------------- the model
def forward(tokens, cfg, weights, dtype=np.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) receives the stream that leaves every layer."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, cfg, w)
    history, latents = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        pre, mix = f"l{i}.", layer["mixer"]
        if layer["type"] == "mingru":
            y = mingru(x, w, pre + "mix.")
        elif layer["type"] == "latent_attention":
            src = mix.get("kv_from")
            y, latents[i] = latent_attention(x, mix, w, pre + "mix.", eps, None if src is None else latents[src])
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(y, w[pre + "norm1"], eps)
        if layer.get("mlp"):
            p, q = w[pre + "mlp.act"]
            y = xielu(x @ w[pre + "mlp.up"].T, p, q) @ w[pre + "mlp.down"].T
            x = x + rms_norm(y, w[pre + "norm2"], eps)
        history.append(x)
        x = depth_average(history, w[pre + "dwa"])
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
