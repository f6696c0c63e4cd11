from .batch import CacheLayout, KVSpec, StepBatch  # noqa: F401
from .engine import BlockManager, LayerStep, LLMEngine, PagedKVCache, Scheduler, Sequence, StatePool  # noqa: F401
