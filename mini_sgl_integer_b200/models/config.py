"""The configuration types the model classes read: the fields of ``minisgl.models.config`` (models/config.py:9-25,
:91-110) that the integer path uses.  The reference's own ``ModelConfig`` (built by ``from_hf``) can be passed
wherever these are expected: only the attributes below are read."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple


@dataclass(frozen=True)
class RotaryConfig:
    head_dim: int
    rotary_dim: int
    max_position: int
    base: float
    scaling: Optional[Dict[str, Any]] = None
    apply_hadamard: bool = True


@dataclass(frozen=True)
class HadamardTransformConfig:
    enabled: bool = False
    block_size: int = 0
    targets: Tuple[str, ...] = ()
    r3_enabled: bool = False


@dataclass(frozen=True)
class ModelConfig:
    num_layers: int
    num_qo_heads: int
    num_kv_heads: int
    head_dim: int
    hidden_size: int
    vocab_size: int
    intermediate_size: int
    rms_norm_eps: float
    rotary_config: RotaryConfig
    tie_word_embeddings: bool = False
    hadamard_transform: HadamardTransformConfig = field(default_factory=HadamardTransformConfig)


# ----------------------------------------------------------------------------- hybrid models in floating point
@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` entries of a vector, entry i paired with entry i + dims / 2."""

    dims: int
    base: float
    scaling: Optional[YarnScaling] = None


@dataclass(frozen=True)
class MinGRUConfig:
    width: int


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                          # unrotated query / key entries per head
    rot_dim: int                      # rotated entries (one key part shared by the heads)
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int] = None      # width of the causal window in keys; None: unbounded
    rot: Optional[RotarySpec] = None
    kv_from: Optional[int] = None     # layer whose latent cache is used instead of an own one


@dataclass(frozen=True)
class DenseMLPConfig:
    ff: int


@dataclass(frozen=True)
class HybridLayerConfig:
    type: str                         # "mingru" or "latent_attention"
    mixer: Any
    mlp: Optional[DenseMLPConfig] = None


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class SefevikConfig:
    """A stack of recurrent and latent-attention layers with output norms and depth averages."""

    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[HybridLayerConfig, ...]
    bigram: Optional[BigramConfig] = None
    architecture: str = "Sefevik"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def attention_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if l.type == "latent_attention")

    @property
    def cache_layers(self) -> Tuple[int, ...]:
        """Layers that own a latent cache."""
        return tuple(i for i in self.attention_layers if self.layers[i].mixer.kv_from is None)

    @property
    def recurrent_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if l.type == "mingru")

    @property
    def max_window(self) -> Optional[int]:
        """Keys behind a token that some layer may still read (itself included); None when a layer has no window, 0
        when no layer attends."""
        windows = [self.layers[i].mixer.window for i in self.attention_layers]
        return None if None in windows else max(windows, default=0)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SefevikConfig":
        if d.get("architecture") != "Sefevik":
            raise ValueError(f"not a Sefevik configuration: architecture {d.get('architecture')!r}")
        layers = tuple(_hybrid_layer(i, l) for i, l in enumerate(d["layers"]))
        for i, l in enumerate(layers):
            src = getattr(l.mixer, "kv_from", None)
            if src is None:
                continue
            if not 0 <= src < i or layers[src].type != "latent_attention" or layers[src].mixer.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {src} does not name an earlier layer with a cache of its own")
            own, other = l.mixer, layers[src].mixer
            if (own.kv_rank, own.rot_dim, own.rot) != (other.kv_rank, other.rot_dim, other.rot):
                raise ValueError(f"layer {i}: kv_rank, rot_dim or rotation differ from layer {src}'s, whose cache it uses")
        big = (d.get("embedding") or {}).get("bigram")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=layers,
                   bigram=BigramConfig(int(big["buckets"]), int(big["mul_prev"]), int(big["mul_cur"])) if big else None)


def _rotary_spec(rot: Optional[Dict[str, Any]]) -> Optional[RotarySpec]:
    if not rot:
        return None
    sc = rot.get("scaling")
    return RotarySpec(int(rot["dims"]), float(rot["base"]),
                      YarnScaling(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None)


def _hybrid_layer(i: int, l: Dict[str, Any]) -> HybridLayerConfig:
    m = l["mixer"]
    if l["type"] == "mingru":
        mixer: Any = MinGRUConfig(int(m["width"]))
    elif l["type"] == "latent_attention":
        size = (m.get("mask") or {}).get("size")
        mixer = LatentAttentionConfig(
            heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
            scale=float(m["scale"]), window=None if size is None else int(size), rot=_rotary_spec(m.get("rot")),
            kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        if mixer.rot is not None and (mixer.rot.dims % 2 or mixer.rot.dims > mixer.rot_dim):
            raise ValueError(f"layer {i}: rotation over {mixer.rot.dims} of {mixer.rot_dim} entries")
        if mixer.window is not None and mixer.window < 1:
            raise ValueError(f"layer {i}: window {mixer.window}")
    else:
        raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
    mlp = l.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    return HybridLayerConfig(l["type"], mixer, DenseMLPConfig(int(mlp["ff"])) if mlp is not None else None)
