from ..registry import Registry  # noqa: F401
from .kv_pool import Int8PagedKVCache, PAGE_SIZE  # noqa: F401
from .ops import (  # noqa: F401
    decode_attention_int8_paged, extend_attention_int8_paged, prefill_attention_int8_paged, qkv_rope_quant_store,
    quantize_per_tensor_int8_ms,
)
from .backend import B200Int8Backend, BaseAttnBackend, BaseAttnMetadata, Int8Metadata  # noqa: F401,E402


# The registry the reference selects backends from with ``--attn`` (attention/__init__.py:20-37); this package
# registers one name per kind of cache.  Inside the reference, the same two lines register one next to "triton_int8".
SUPPORTED_ATTENTION_BACKENDS = Registry("Attention Backend")


@SUPPORTED_ATTENTION_BACKENDS.register("b200_int8")
def create_b200_int8_backend(config, kvcache):
    return B200Int8Backend(config, kvcache)


@SUPPORTED_ATTENTION_BACKENDS.register("b200_hybrid")
def create_b200_hybrid_backend(config, kvcache):
    from .hybrid_backend import B200HybridBackend
    return B200HybridBackend(config, kvcache)


def create_attention_backend(backend: str, config, kvcache):
    """attention/__init__.py:66-89 for the backends of this package."""
    return SUPPORTED_ATTENTION_BACKENDS[backend](config, kvcache)
