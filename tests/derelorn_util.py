"""Small Derelorn configurations and weights for the tests, in the form of config.json and of a checkpoint."""
from __future__ import annotations

import torch

from mini_sgl_integer_b200.models.config import DerelornConfig
from mini_sgl_integer_b200.models.derelorn import random_weights
from tests.sefevik_util import logit_error, numpy_weights, write_model  # noqa: F401  (shared helpers)


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def mlstm(heads, dim, vdim, ff=None, cap=15.0):
    return layer("mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, ff)


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return layer("delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, ff)


def attn(heads, kv_heads, dim, vdim, window, scale):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return m


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(left, right, ff=None):
    return layer("parallel", {"left": left, "right": right}, ff)


def model(vocab, width, layers, loop=None, eps=1e-5):
    d = {"architecture": "Derelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# the scales of the scores are large: single keys stand out, so that a wrong, missing or extra key shows in the logits
CONFIGS = {
    "mixed": model(123, 80, [parallel(attn(6, 2, 16, 24, 21, 0.9), mamba(6, 16, 24, 2, 4, 3), 72), mlstm(3, 24, 16, 40, cap=9.0),
                             delta(6, 2, 24, 16, 3, 56), mlstm(2, 40, 48)], loop=(1, 3, 3)),
    "odd sizes": model(57, 50, [delta(3, 1, 11, 13, 2, 37), parallel(attn(3, 3, 9, 7, 34, 1.0), mamba(5, 6, 10, 1, 5, 2), 19), mlstm(5, 7, 9, 21, cap=4.5),
                                delta(2, 2, 20, 6, 1)], eps=1e-3),
    "loop over everything": model(64, 48, [parallel(attn(4, 1, 24, 16, 1, 0.7), mamba(2, 40, 8, 2, 1, 2)), delta(2, 1, 16, 32, 4, 48)], loop=(0, 2, 2)),
    "loop at the end, once": model(90, 64, [mlstm(4, 16, 24, 64), parallel(attn(8, 4, 16, 16, 90, 0.8), mamba(4, 24, 16, 4, 3, 1), 40)], loop=(1, 2, 1)),
    "wide heads": model(70, 128, [mlstm(2, 144, 136, 96), parallel(attn(40, 2, 136, 40, 37, 0.25), mamba(2, 136, 72, 1, 4, 2)),
                                  delta(2, 1, 260, 72, 4), parallel(attn(3, 1, 72, 200, None, 0.3), mamba(3, 8, 130, 3, 2, 1), 64)]),
    "one layer": model(33, 24, [mlstm(1, 8, 8, 16)]),
}


def make_weights(cfg: dict, seed: int) -> dict:
    """bf16 weights; the first head of every mlstm layer writes weakly, so that its read-outs stay under the normaliser's floor
    and are as small as the norms' eps."""
    sd = random_weights(DerelornConfig.from_dict(cfg), seed)
    for i, l in enumerate(cfg["layers"]):
        if l["type"] == "mlstm":
            sd[f"l{i}.mix.i.b"][0] -= 6.0
    return sd


def attention_window(cfg: dict):
    w = [(l["mixer"]["left"].get("mask") or {}).get("size") for l in cfg["layers"] if l["type"] == "parallel"]
    return None if None in w else max(w, default=0)


def float_weights(sd: dict) -> dict:
    return {k: v.to(torch.float64).numpy() for k, v in sd.items()}
