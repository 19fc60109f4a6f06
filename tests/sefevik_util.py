"""Small Sefevik configurations and weights for the tests, in the form of config.json and of a checkpoint."""
from __future__ import annotations

import json
import os
import struct

import numpy as np
import torch

from mini_sgl_integer_b200.models.config import SefevikConfig
from mini_sgl_integer_b200.models.sefevik import random_weights

YARN = {"factor": 4.0, "original": 64, "fast": 6.0, "slow": 1.0}


def gru(width, ff=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def mla(heads, dim, rot_dim, vdim, kv_rank, window, scale, ff=None, kv_from=None, base=10000.0, scaling=YARN):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def model(vocab, width, layers, bigram=(29, 7, 3), eps=1e-5):
    d = {"architecture": "Sefevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if bigram:
        d["embedding"] = {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}
    return d


# the scales are large: single scores stand out, so that a wrong, missing or extra key shows in the logits
CONFIGS = {
    "mixed": model(131, 72, [gru(40, 88), mla(3, 24, 12, 16, 40, 37, 0.6, ff=104), gru(96), mla(5, 16, 12, 8, 40, 70, 0.7, ff=56, kv_from=1),
                             mla(2, 8, 4, 32, 16, 18, 0.9), gru(56, 24)]),
    "odd sizes": model(61, 50, [mla(2, 11, 6, 9, 22, 21, 0.8, ff=37, base=500.0), gru(33, 19), mla(1, 5, 6, 7, 22, 40, 0.9, kv_from=0, base=500.0)],
                       bigram=(11, 5, 2), eps=1e-3),
    "attention only, no bigram, full and single-token windows": model(
        97, 64, [mla(4, 16, 8, 16, 32, None, 0.5, ff=64, scaling=None), mla(17, 8, 8, 8, 24, 1, 0.6, ff=40, scaling=None),
                 mla(6, 16, 8, 24, 32, 16, 0.7, kv_from=0, scaling=None)], bigram=None),
    "recurrence only": model(80, 40, [gru(64, 48), gru(24), gru(136, 16)], bigram=(1, 3, 5)),
    "wide heads": model(70, 128, [mla(20, 32, 16, 24, 128, 90, 0.3, ff=96), mla(70, 16, 16, 8, 128, 33, 0.35, kv_from=0), gru(200, 64)]),
    "one layer": model(33, 24, [mla(1, 8, 2, 8, 8, 9, 1.0, ff=16, scaling={"factor": 2.0, "original": 16, "fast": 4.0, "slow": 2.0})]),
}


def make_weights(cfg: dict, seed: int) -> dict:
    """bf16 weights; recurrent gates are biased towards long memory."""
    sd = random_weights(SefevikConfig.from_dict(cfg), seed)
    for i, l in enumerate(cfg["layers"]):
        if l["type"] == "mingru":
            sd[f"l{i}.mix.z.b"] = (sd[f"l{i}.mix.z.b"].float() - 3.0).to(torch.bfloat16)
    return sd


def numpy_weights(sd: dict) -> dict:
    return {k: v.float().numpy() for k, v in sd.items()}


def write_model(path: str, cfg: dict, sd: dict) -> None:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, data = {}, b""
    for k, v in sd.items():
        raw = v.contiguous().view(torch.int16).numpy().tobytes()
        head[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + data)


def logit_error(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: root mean square of the difference with its mean taken off, relative to that of the row."""
    d = got.astype(np.float64) - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1) / (w ** 2).mean(-1))
