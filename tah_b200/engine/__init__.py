"""Inference engines: paged KV (per iteration depth, per layer), recurrent state, scheduling, CUDA-graph ticks."""
from tah_b200.engine.base import DecodeEngine, GenerationResult
from tah_b200.engine.engine import TaHEngine, get_engine
from tah_b200.engine.hybrid import HybridEngine, StepEntry
from tah_b200.engine.kv_cache import CacheGeometry, LayerKV, PagedKVCache, RecurrentState

__all__ = ["DecodeEngine", "TaHEngine", "HybridEngine", "StepEntry", "GenerationResult", "get_engine", "PagedKVCache",
           "CacheGeometry", "LayerKV", "RecurrentState"]
