"""Verozen: a decoder with norms after the residual sums whose layers mix tokens by gated linear attention, by sigmoid
attention or by retention, with routed experts for the feed-forward and a small per-layer token input.

``VerozenConfig`` reads the checkpoint's config.json.  The residual stream is float32; ``dtype`` is the type of weights,
activations and K/V caches (bfloat16 for serving, float32 for exact work)."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Callable, Optional

import torch
import torch.nn as nn

from ..engine.batch import CacheLayout, StepBatch
from ..layers import mixers as ops
from ..layers.sequence_mixers import (GatedLinearMixer, GroupNorm, ParallelMixer, RetentionMixer, RoutedExperts, SigmoidAttentionMixer,
                                      TokenSideInput)


@dataclass
class VerozenConfig:
    vocab: int
    width: int
    layers: list           # dicts with "type", "mixer" (of a gla layer with its gate's "rank") and "mlp" (or None)
    norm_groups: int
    eps: float
    alpha: float           # of the residual sums ahead of the norms
    side_dim: int          # per-layer token input

    @classmethod
    def from_dict(cls, c: dict) -> "VerozenConfig":
        cfg = cls(int(c["vocab"]), int(c["width"]), list(c["layers"]), int(c["norm"]["groups"]), float(c["norm"]["eps"]),
                  float(c["postln_alpha"]), int(c["token_side"]["dim"]))
        for i, lay in enumerate(cfg.layers):
            if lay["type"] not in ("gla", "attention", "retention"):
                raise ValueError(f"layer {i}: unknown mixer `{lay['type']}`")
            if lay["type"] == "gla" and "rank" not in lay["mixer"]:
                raise ValueError(f"layer {i}: the rank of the decay's projection is not known")
            if lay["type"] == "attention" and lay["mixer"]["vdim"] != lay["mixer"]["dim"]:
                raise ValueError(f"layer {i}: the values are the keys, so vdim must be dim")
            if lay.get("mlp") is not None and lay["mlp"]["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward `{lay['mlp']['kind']}`")
        return cfg

    @staticmethod
    def complete(c: dict, shapes: dict) -> dict:
        """The rank of a gla layer's decay projection is the first size of its tensor."""
        c = copy.deepcopy(c)
        for i, lay in enumerate(c["layers"]):
            if lay["type"] == "gla":
                lay["mixer"]["rank"] = shapes[f"l{i}.mix.a1"][0]
        return c


def _mixer(cfg: VerozenConfig, kind: str, m: dict, dtype, device) -> nn.Module:
    if kind == "gla":
        return GatedLinearMixer(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], rank=m["rank"], tau=m["tau"], eps=cfg.eps, dtype=dtype, device=device)
    rot = dict(rot_base=m["rot"]["base"], rot_dims=m["rot"]["dims"])
    if kind == "attention":
        return SigmoidAttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], interleaved=True, scale=m["scale"], eps=cfg.eps,
                                     device=device, **rot)
    return RetentionMixer(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=m["decay"], eps=cfg.eps, device=device, **rot)


class VerozenLayer(nn.Module):
    def __init__(self, cfg: VerozenConfig, index: int, *, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        spec = cfg.layers[index]
        self.alpha = cfg.alpha
        self.mixer = ParallelMixer(cfg.width, {"only": _mixer(cfg, spec["type"], spec["mixer"], dtype, device)}, beta=cfg.alpha,
                                   prefixes={"only": ""}, **kw)
        self.norm1 = GroupNorm(cfg.width, cfg.norm_groups, cfg.eps, **kw)
        f = spec.get("mlp")
        self.mlp = self.norm2 = None
        if f is not None:
            r = f["router"]
            self.mlp = RoutedExperts(cfg.width, int(f["expert"]["ff"]), experts=r["experts"], top=r["top"], groups=r["groups"]["count"],
                                     keep=r["groups"]["keep"], scale=r["scale"], **kw)
            self.norm2 = GroupNorm(cfg.width, cfg.norm_groups, cfg.eps, **kw)
        self.side = TokenSideInput(cfg.width, cfg.side_dim, index * cfg.side_dim, cfg.eps, **kw)

    def checkpoint(self, prefix: str) -> dict:
        out = self.mixer.checkpoint(prefix + "mix.")
        out[prefix + "norm1"] = self.norm1.weight
        if self.mlp is not None:
            out.update(self.mlp.checkpoint(prefix + "mlp."))
            out[prefix + "norm2"] = self.norm2.weight
        out.update(self.side.checkpoint(prefix + "side."))
        return out

    def forward(self, x, h, layer_step, tokens, table):
        """Advances the float32 stream ``x`` in place; ``h`` is its rounding, and so is what is returned."""
        self.mixer(x, h, layer_step)
        h = self.norm1(x)
        if self.mlp is not None:
            h = self.norm2(x, self.mlp(h), self.alpha)
        return self.side(x, h, tokens, table)


class VerozenForCausalLM(nn.Module):
    tp_size, tp_rank = 1, 0
    delegates_attention = False

    def __init__(self, cfg: VerozenConfig, *, device="cpu", dtype=torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"Verozen runs in bfloat16 or float32, not {dtype}")
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device(device)
        self.vocab_size = cfg.vocab
        for name, shape in (("embed", (cfg.vocab, cfg.width)), ("head", (cfg.vocab, cfg.width)),
                            ("side_embed", (cfg.vocab, len(cfg.layers) * cfg.side_dim))):
            self.register_buffer(name, torch.zeros(*shape, dtype=dtype, device=device), persistent=False)
        self.layers = nn.ModuleList([VerozenLayer(cfg, i, dtype=dtype, device=device) for i in range(len(cfg.layers))])
        self.final_norm = GroupNorm(cfg.width, cfg.norm_groups, cfg.eps, dtype=dtype, device=device)

    # -------------------------------------------------------------- loading and caching
    def checkpoint_tensors(self) -> dict[str, torch.Tensor]:
        """Checkpoint name -> the view it is copied into (parts of merged weights among them)."""
        out = {"embed": self.embed, "head": self.head, "side.embed": self.side_embed, "final.norm": self.final_norm.weight}
        for i, layer in enumerate(self.layers):
            out.update(layer.checkpoint(f"l{i}."))
        return out

    def cache_layout(self) -> CacheLayout:
        return CacheLayout([layer.mixer.kv_spec() for layer in self.layers], [layer.mixer.state_shapes() for layer in self.layers])

    # -------------------------------------------------------------- one step
    def forward_step(self, batch: StepBatch, layer_step: Callable[[int], object], rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Runs the step's tokens from the caches and states that earlier steps left; returns the final norm of the
        given rows (all tokens if None)."""
        x = torch.empty(batch.num_tokens, self.cfg.width, dtype=torch.float32, device=self.device)
        ops.stream_add(x, batch.tokens, self.embed, None, False)
        h = nn.functional.embedding(batch.tokens, self.embed)
        for i, layer in enumerate(self.layers):
            h = layer(x, h, layer_step(i), batch.tokens, self.side_embed)
        return self.final_norm.rows(x, rows)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return ops.linear(hidden, self.head, torch.float32)

    @torch.no_grad()
    def greedy_tokens(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits(hidden).argmax(dim=-1)
