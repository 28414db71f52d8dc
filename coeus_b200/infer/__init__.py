"""Inference: paged KV cache, sampling, and the generation engines."""
from .engine import InferenceEngine, make_engine  # noqa: F401
from .kv_cache import PagedKVCache, SequenceState  # noqa: F401
