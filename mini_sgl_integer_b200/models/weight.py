"""Checkpoint reading: safetensors files (one, or the shards that model.safetensors.index.json lists) to host tensors.

A file is an 8-byte little-endian header length, a JSON header name -> {dtype, shape, data_offsets}, then the data; it is
memory-mapped, so a tensor's bytes are read when it is copied to the device.
"""
from __future__ import annotations

import json
import mmap
import os
import struct
from typing import Any, Dict

import torch

_DTYPES = {"F64": torch.float64, "F32": torch.float32, "F16": torch.float16, "BF16": torch.bfloat16, "I64": torch.int64,
           "I32": torch.int32, "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        head = f.read(8)
        if len(head) != 8:
            raise ValueError(f"{path}: not a safetensors file")
        n = struct.unpack("<Q", head)[0]
        size = os.fstat(f.fileno()).st_size
        if n > size - 8:
            raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
        entries = json.loads(f.read(n))
        data = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_COPY)
    out: Dict[str, torch.Tensor] = {}
    for name, e in entries.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in _DTYPES:
            raise ValueError(f"{path}: tensor {name} has unsupported dtype {e['dtype']}")
        dtype, shape, (lo, hi) = _DTYPES[e["dtype"]], tuple(e["shape"]), e["data_offsets"]
        count = 1
        for d in shape:
            count *= d
        if hi - lo != count * dtype.itemsize or 8 + n + hi > size:
            raise ValueError(f"{path}: tensor {name} does not fit its data range")
        if count == 0:
            out[name] = torch.empty(shape, dtype=dtype)
        elif (8 + n + lo) % dtype.itemsize:
            out[name] = torch.frombuffer(bytearray(data[8 + n + lo:8 + n + hi]), dtype=dtype).reshape(shape)
        else:
            out[name] = torch.frombuffer(data, dtype=dtype, count=count, offset=8 + n + lo).reshape(shape)
    return out


def load_checkpoint(model_dir: str) -> Dict[str, torch.Tensor]:
    index = os.path.join(model_dir, "model.safetensors.index.json")
    if os.path.exists(index):
        with open(index) as f:
            files = sorted(set(json.load(f)["weight_map"].values()))
    else:
        files = ["model.safetensors"]
    out: Dict[str, torch.Tensor] = {}
    for name in files:
        out.update(read_safetensors(os.path.join(model_dir, name)))
    return out


def load_config_dict(model_dir: str) -> Dict[str, Any]:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def architecture_of(config: Dict[str, Any]) -> str:
    """``architecture``, or the one entry of Hugging Face's ``architectures``."""
    if "architecture" in config:
        return str(config["architecture"])
    names = config.get("architectures") or []
    if len(names) != 1:
        raise ValueError("config.json names no architecture")
    return str(names[0])
