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
class MLSTMConfig:
    """Matrix memory with exponential gates."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float                   # log gates are cap * tanh(pre / cap)


@dataclass(frozen=True)
class GatedDeltaConfig:
    """Matrix memory written by the delta rule, one decay per head."""

    heads: int
    kv_heads: int                     # query / key heads
    dim: int
    vdim: int
    conv: int                         # taps of the short convolutions


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int                       # of B and C
    conv: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class GroupedAttentionConfig:
    """Softmax attention whose query heads share key heads; q and k normed over the whole projection, no rotation."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None


@dataclass(frozen=True)
class ParallelConfig:
    """Two mixers that read the same input."""

    left: GroupedAttentionConfig
    right: Mamba2Config


@dataclass(frozen=True)
class DenseMLPConfig:
    ff: int


@dataclass(frozen=True)
class HybridLayerConfig:
    type: str                         # "mingru", "latent_attention", "mlstm", "delta", "parallel"
    mixer: Any
    mlp: Optional[DenseMLPConfig] = None


@dataclass(frozen=True)
class RunMemory:
    """What one run of a layer keeps per sequence.  ``planes``: (heads, values per head) of the rows it stores per token in
    pages, keys first; ``value_prefix``: values are the first entries of the key row.  ``state``: name -> shape, fp32."""

    planes: Tuple[Tuple[int, int], ...] = ()
    value_prefix: Optional[int] = None
    state: Tuple[Tuple[str, Tuple[int, ...]], ...] = ()


def mixer_memory(m: Any) -> RunMemory:
    pad = lambda n: (n + 7) // 8 * 8                                   # values of a head start on 16-byte boundaries
    if isinstance(m, MinGRUConfig):
        return RunMemory(state=(("s", (m.width,)),))
    if isinstance(m, LatentAttentionConfig):
        return RunMemory() if m.kv_from is not None else RunMemory(((1, m.kv_rank + m.rot_dim),), m.kv_rank)
    if isinstance(m, GroupedAttentionConfig):
        return RunMemory(((m.kv_heads, m.dim), (m.kv_heads, m.vdim)))
    if isinstance(m, MLSTMConfig):
        return RunMemory(state=(("S", (m.heads, m.dim, pad(m.vdim))), ("n", (m.heads, m.dim + 1))))
    if isinstance(m, GatedDeltaConfig):
        return RunMemory(state=(("S", (m.heads, m.dim, pad(m.vdim))), ("conv", (m.conv - 1, 2 * m.kv_heads * m.dim + m.heads * m.vdim))))
    if isinstance(m, Mamba2Config):
        return RunMemory(state=(("S", (m.heads, m.state, pad(m.vdim))), ("conv", (m.conv - 1, m.inner + 2 * m.groups * m.state))))
    if isinstance(m, ParallelConfig):
        a, b = mixer_memory(m.left), mixer_memory(m.right)
        return RunMemory(a.planes + b.planes, state=a.state + b.state)
    raise TypeError(f"no cache is known for {type(m).__name__}")


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
        return widest_window([self.layers[i].mixer.window for i in self.attention_layers])

    @property
    def memory(self) -> Tuple[RunMemory, ...]:
        return tuple(mixer_memory(l.mixer) for l in self.layers)

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


def widest_window(windows) -> Optional[int]:
    """Keys behind a token that some layer may still read (itself included); None when a layer has no window, 0 when no
    layer attends."""
    return None if None in windows else max(windows, default=0)


@dataclass(frozen=True)
class LoopConfig:
    """Layers start .. stop - 1 run ``times`` times in a row."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    layer: int
    begins: Optional[int] = None      # the pass of the loop that begins with this run


@dataclass(frozen=True)
class DerelornConfig:
    """A stack of matrix memories and windowed attention, normed in front of and behind every sublayer; some layers may be
    run several times."""

    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[HybridLayerConfig, ...]
    loop: Optional[LoopConfig] = None
    architecture: str = "Derelorn"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> Tuple[LayerRun, ...]:
        """Layers in the order of execution.  Every run has a cache and a state of its own."""
        n, l = len(self.layers), self.loop
        if l is None:
            return tuple(LayerRun(i) for i in range(n))
        passes = [LayerRun(i, t if i == l.start else None) for t in range(l.times) for i in range(l.start, l.stop)]
        return tuple([LayerRun(i) for i in range(l.start)] + passes + [LayerRun(i) for i in range(l.stop, n)])

    @property
    def memory(self) -> Tuple[RunMemory, ...]:
        return tuple(mixer_memory(self.layers[r.layer].mixer) for r in self.runs)

    @property
    def cache_layers(self) -> Tuple[int, ...]:
        """Runs that own a paged cache."""
        return tuple(i for i, m in enumerate(self.memory) if m.planes)

    @property
    def max_window(self) -> Optional[int]:
        return widest_window([l.mixer.left.window for l in self.layers if l.type == "parallel"])

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "DerelornConfig":
        if d.get("architecture") != "Derelorn":
            raise ValueError(f"not a Derelorn configuration: architecture {d.get('architecture')!r}")
        layers = tuple(_hybrid_layer(i, l) for i, l in enumerate(d["layers"]))
        for i, l in enumerate(layers):
            if l.type not in ("mlstm", "delta", "parallel"):
                raise ValueError(f"layer {i}: the design has no mixer {l.type!r}")
        loop = d.get("loop")
        if loop:
            loop = LoopConfig(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"loop over layers {loop.start} .. {loop.stop - 1}, {loop.times} times, of {len(layers)}")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=layers, loop=loop or None)


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
    elif l["type"] == "mlstm":
        mixer = MLSTMConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
        if not mixer.gate_cap > 0:
            raise ValueError(f"layer {i}: gate_cap {mixer.gate_cap}")
    elif l["type"] == "delta":
        mixer = GatedDeltaConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        _check_shared(i, mixer.heads, mixer.kv_heads)
        _check_taps(i, mixer.conv)
    elif l["type"] == "parallel":
        mixer = ParallelConfig(_grouped_attention(i, m["left"]), _mamba2(i, m["right"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
    mlp = l.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    return HybridLayerConfig(l["type"], mixer, DenseMLPConfig(int(mlp["ff"])) if mlp is not None else None)


def _check_shared(i: int, heads: int, shared: int) -> None:
    if shared < 1 or heads % shared:
        raise ValueError(f"layer {i}: {heads} heads cannot share {shared}")


def _check_taps(i: int, taps: int) -> None:
    if taps < 1:
        raise ValueError(f"layer {i}: a convolution of {taps} taps")


def _grouped_attention(i: int, m: Dict[str, Any]) -> GroupedAttentionConfig:
    size = (m.get("mask") or {}).get("size")
    c = GroupedAttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), None if size is None else int(size))
    _check_shared(i, c.heads, c.kv_heads)
    if c.window is not None and c.window < 1:
        raise ValueError(f"layer {i}: window {c.window}")
    return c


def _mamba2(i: int, m: Dict[str, Any]) -> Mamba2Config:
    c = Mamba2Config(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m["norm_groups"]))
    _check_shared(i, c.heads, c.groups)
    _check_taps(i, c.conv)
    if c.norm_groups < 1 or c.inner % c.norm_groups:
        raise ValueError(f"layer {i}: {c.inner} values cannot be normed in {c.norm_groups} parts")
    return c
