"""Architecture name -> how the engine configures, loads, caches and runs a model (models/register.py and
models/weight.py:55-138 of the reference play this part)."""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from ..registry import Registry
from .config import DerelornConfig, HadamardTransformConfig, ModelConfig, RotaryConfig, SefevikConfig

SUPPORTED_MODELS = Registry("Model architecture")


class ModelEntry:
    """What the engine asks of an architecture."""

    dtypes: tuple = ()
    library: str = "int"                     # the kernel library it runs on
    backend: str = ""                        # name in SUPPORTED_ATTENTION_BACKENDS

    def parse_config(self, d: Dict[str, Any]) -> Any:
        raise NotImplementedError

    def vocab_size(self, config) -> int:
        return config.vocab_size

    def window(self, config) -> Optional[int]:
        """Keys that stay readable behind a token, or None for all of them."""
        return None

    def needs_pages(self, config) -> bool:
        return True

    def create(self, config, weights: Dict[str, torch.Tensor], dtype: torch.dtype, device, max_len: int):
        """The model with its weights on the device; consumes ``weights``."""
        raise NotImplementedError

    def create_cache(self, config, num_pages: int, num_slots: int, dtype: torch.dtype, device):
        raise NotImplementedError

    def check_status(self) -> None:
        """Raises when a kernel of the last steps gave up waiting; synchronises with the device."""


class HybridEntry(ModelEntry):
    """Floating-point designs over ``HybridCache``."""

    dtypes = (torch.bfloat16, torch.float32)
    library = "float"
    backend = "b200_hybrid"

    def window(self, config):
        return config.max_window

    def needs_pages(self, config):
        return bool(config.cache_layers)

    def create_cache(self, config, num_pages, num_slots, dtype, device):
        from ..kvcache.hybrid_pool import HybridCache
        return HybridCache(config, num_pages, num_slots, dtype, device)

    def check_status(self):
        from ..kernel.float_ops import check_status
        check_status()


@SUPPORTED_MODELS.register("Sefevik")
class SefevikEntry(HybridEntry):
    def parse_config(self, d):
        return SefevikConfig.from_dict(d)

    def create(self, config, weights, dtype, device, max_len):
        from .sefevik import SefevikForCausalLM
        model = SefevikForCausalLM(config, dtype, device, max_position=max_len)
        model.load_state_dict(weights)
        return model


@SUPPORTED_MODELS.register("Derelorn")
class DerelornEntry(HybridEntry):
    def parse_config(self, d):
        return DerelornConfig.from_dict(d)

    def create(self, config, weights, dtype, device, max_len):
        from .derelorn import DerelornForCausalLM
        model = DerelornForCausalLM(config, dtype, device)
        model.load_state_dict(weights)
        return model


@SUPPORTED_MODELS.register("Qwen3ForCausalLM")
class Qwen3IntegerEntry(ModelEntry):
    """int8 checkpoints of Qwen3 (``weight`` int8 + ``weight_scale``), run in integers whatever the asked dtype."""

    dtypes = (torch.bfloat16,)
    backend = "b200_int8"

    def parse_config(self, d):
        heads = int(d["num_attention_heads"])
        scaling = d.get("rope_scaling")
        return ModelConfig(
            num_layers=int(d["num_hidden_layers"]), num_qo_heads=heads, num_kv_heads=int(d.get("num_key_value_heads", heads)),
            head_dim=int(d.get("head_dim") or d["hidden_size"] // heads), hidden_size=int(d["hidden_size"]), vocab_size=int(d["vocab_size"]),
            intermediate_size=int(d["intermediate_size"]), rms_norm_eps=float(d["rms_norm_eps"]),
            rotary_config=RotaryConfig(int(d.get("head_dim") or d["hidden_size"] // heads), int(d.get("head_dim") or d["hidden_size"] // heads),
                                       int(d["max_position_embeddings"]), float(d["rope_theta"]), scaling),
            tie_word_embeddings=bool(d.get("tie_word_embeddings", False)), hadamard_transform=_hadamard_of(d))

    def create(self, config, weights, dtype, device, max_len):
        from ..distributed import set_tp_info, try_get_tp_info
        from .integer import Qwen3ForCausalLMInteger
        if try_get_tp_info() is None:
            set_tp_info(0, 1)
        model = Qwen3ForCausalLMInteger(config)
        model.load_state_dict(_merge_qwen3(weights, dtype, device))
        return model

    def create_cache(self, config, num_pages, num_slots, dtype, device):
        from ..attention import Int8PagedKVCache
        pool = Int8PagedKVCache(config.num_kv_heads, config.num_layers, config.head_dim, num_pages + 1, device)
        pool.spare_page, pool.spare_slot = num_pages, num_slots
        return pool

    def check_status(self):
        from .qwen3_integer import check_device_status
        check_device_status()


def _hadamard_of(d: Dict[str, Any]) -> HadamardTransformConfig:
    """The input rotation of a compressed-tensors checkpoint (models/config.py:27-88): the targets and block of its
    Hadamard group."""
    groups = ((d.get("quantization_config") or {}).get("transform_config") or {}).get("config_groups") or {}
    targets, block, r3 = [], 0, False
    for name, g in groups.items():
        if g.get("type") != "hadamard":
            continue
        inputs = [a for a in g.get("apply", []) if a.get("location") == "input"]
        if inputs:
            block = int(g.get("head_dim") or block)
            for a in inputs:
                targets.extend(a.get("targets", []))
        r3 = r3 or name == "R3"
    return HadamardTransformConfig(enabled=bool(targets), block_size=block, targets=tuple(targets), r3_enabled=r3)


_MERGED = {"qkv_proj": ("q_proj", "k_proj", "v_proj"), "gate_up_proj": ("gate_proj", "up_proj")}


def _merge_qwen3(weights: Dict[str, torch.Tensor], dtype: torch.dtype, device) -> Dict[str, torch.Tensor]:
    """Hugging Face keys to the model's: q / k / v and gate / up stacked along the output (weights and channel scales),
    floating-point tensors other than scales in ``dtype``."""
    out: Dict[str, torch.Tensor] = {}
    part_of = {p: (m, i, len(ps)) for m, ps in _MERGED.items() for i, p in enumerate(ps)}
    waiting: Dict[str, list] = {}
    for key in list(weights):
        t = weights.pop(key)
        keep = t.dtype == torch.int8 or key.endswith("_scale")
        t = t.to(device) if keep else t.to(device=device, dtype=dtype)
        names = key.split(".")
        hit = next((n for n in names if n in part_of), None)
        if hit is None:
            out[key] = t
            continue
        merged, i, n = part_of[hit]
        new_key = ".".join(merged if x == hit else x for x in names)
        slots = waiting.setdefault(new_key, [None] * n)
        slots[i] = t
        if all(x is not None for x in slots):
            out[new_key] = torch.cat(waiting.pop(new_key))
    if waiting:
        raise KeyError(f"incomplete merged tensors: {sorted(waiting)}")
    return out
