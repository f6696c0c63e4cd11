"""Which model class a checkpoint's config.json names, and how to build and load it."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Optional

import torch

from ..utils.loader import load_model, tensor_shapes
from .qwen3_quantized import Qwen3Config, Qwen3QuantizedForCausalLM
from .vemedra import VemedraConfig, VemedraForCausalLM
from .verozen import VerozenConfig, VerozenForCausalLM


@dataclass(frozen=True)
class ModelEntry:
    config: Callable[[dict], object]        # config.json as a dict -> configuration
    build: Callable[..., torch.nn.Module]   # (configuration, device=, dtype=) -> model with empty weights
    dtypes: tuple                           # what the model's kernels run in
    libraries: tuple                        # kernel libraries it needs (names in csrc.build)
    prepare: Callable[[torch.nn.Module], None] = lambda model: None   # after loading
    # config.json and {tensor name: shape} -> config.json with the sizes that only the tensors give
    complete: Optional[Callable[[dict, dict], dict]] = None


MODELS: dict[str, ModelEntry] = {
    "Qwen3ForCausalLM": ModelEntry(Qwen3Config.from_dict, Qwen3QuantizedForCausalLM.from_config, (torch.bfloat16, torch.float16),
                                   ("LIB_PATH",), lambda model: model.fuse_projections()),
    "Verozen": ModelEntry(VerozenConfig.from_dict, VerozenForCausalLM, (torch.bfloat16, torch.float32), ("MIXERS_PATH", "MOE_PATH"),
                          complete=VerozenConfig.complete),
    "Vemedra": ModelEntry(VemedraConfig.from_dict, VemedraForCausalLM, (torch.bfloat16, torch.float32), ("MIXERS_PATH",)),
}


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json")) as fh:
        return json.load(fh)


def model_class(config: dict) -> ModelEntry:
    """By ``architecture``, or by the first entry of ``architectures`` as Hugging Face writes it."""
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in MODELS:
        raise ValueError(f"no model for architecture `{name}`; known: {', '.join(sorted(MODELS))}")
    return MODELS[name]


def build_model(path: str, *, device="cuda:0", dtype=torch.bfloat16) -> torch.nn.Module:
    """The model of checkpoint folder ``path`` with its weights, ready for the engine."""
    config = read_config(path)
    entry = model_class(config)
    if dtype not in entry.dtypes:
        raise TypeError(f"this model runs in {', '.join(str(d) for d in entry.dtypes)}, not {dtype}")
    if entry.complete is not None:
        config = entry.complete(config, tensor_shapes(path))
    model = entry.build(entry.config(config), device=device, dtype=dtype)
    load_model(model, path)
    entry.prepare(model)
    return model
