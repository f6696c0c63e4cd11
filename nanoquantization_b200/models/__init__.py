from .qwen3_quantized import (Qwen3Config, Qwen3QuantizedAttention, Qwen3QuantizedBlock, Qwen3QuantizedForCausalLM,  # noqa: F401
                              Qwen3QuantizedMLP, Qwen3QuantizedModel, RMSNorm, RotaryCache, QWEN3_SHAPES)
from .vemedra import VemedraConfig, VemedraForCausalLM  # noqa: F401
from .verozen import VerozenConfig, VerozenForCausalLM  # noqa: F401
from .registry import MODELS, build_model, model_class, read_config  # noqa: F401
