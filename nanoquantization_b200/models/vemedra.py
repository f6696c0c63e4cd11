"""Vemedra: a decoder whose layers mix tokens by a minGRU or by chunked attention beside retention, with a short
causal convolution ahead of every sub-layer and a stretch of layers that runs several times with shared weights.

``VemedraConfig`` reads the checkpoint's config.json.  A *run* is one pass through one layer: a looped layer has as
many runs as passes, and each run has its own cache entry and states.  The residual stream is float32; ``dtype`` is
the type of weights, activations and K/V caches (bfloat16 for serving, float32 for exact work)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional

import torch
import torch.nn as nn

from ..engine.batch import CacheLayout, StepBatch
from ..layers import mixers as ops
from ..layers.sequence_mixers import AttentionMixer, ClampedGLU, ConvNorm, MinGRUMixer, ParallelMixer, RetentionMixer


@dataclass
class VemedraConfig:
    vocab: int
    width: int
    layers: list           # dicts with "type", "mixer" and "mlp" (or None)
    taps: int
    eps: float
    loop_start: int = 0    # layers loop_start .. loop_stop - 1 run loop_times times in a row
    loop_stop: int = 0
    loop_times: int = 0

    @classmethod
    def from_dict(cls, c: dict) -> "VemedraConfig":
        loop = c.get("loop") or {"start": 0, "stop": 0, "times": 0}
        cfg = cls(int(c["vocab"]), int(c["width"]), list(c["layers"]), int(c["canon"]["taps"]), float(c["norm"]["eps"]),
                  int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= cfg.loop_start <= cfg.loop_stop <= len(cfg.layers):
            raise ValueError(f"loop over layers {cfg.loop_start}..{cfg.loop_stop} of {len(cfg.layers)}")
        for i, lay in enumerate(cfg.layers):
            if lay["type"] not in ("mingru", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer `{lay['type']}`")
            if lay.get("mlp") is not None and lay["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward `{lay['mlp']['kind']}`")
        return cfg

    def runs(self) -> list[tuple[int, Optional[int]]]:
        """(layer, pass) in the order of execution; the pass is given at the first layer of each pass only."""
        out: list[tuple[int, Optional[int]]] = [(i, None) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            out += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return out + [(i, None) for i in range(self.loop_stop, len(self.layers))]


class VemedraLayer(nn.Module):
    def __init__(self, cfg: VemedraConfig, spec: dict, *, dtype, device):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        m = spec["mixer"]
        if spec["type"] == "mingru":
            self.mixer = MinGRUMixer(cfg.width, int(m["width"]), **kw)
        else:
            a, r = m["left"], m["right"]
            self.mixer = ParallelMixer(cfg.width, {
                "left": AttentionMixer(heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], vdim=a["vdim"], chunk=a["mask"]["size"],
                                       rot_base=a["rot"]["base"], rot_dims=a["rot"]["dims"], scale=a["scale"], softcap=a["softcap"],
                                       out_scale=m["left_scale"], device=device),
                "right": RetentionMixer(heads=r["heads"], dim=r["dim"], vdim=r["vdim"], decay=r["decay"], eps=cfg.eps,
                                        out_scale=m["right_scale"], device=device)}, **kw)
        self.norm1 = ConvNorm(cfg.width, cfg.taps, cfg.eps, **kw)
        f = spec.get("mlp")
        self.mlp = None if f is None else ClampedGLU(cfg.width, int(f["ff"]), f["limit"], **kw)
        self.norm2 = None if f is None else ConvNorm(cfg.width, cfg.taps, cfg.eps, **kw)

    def state_shapes(self) -> dict:
        out = dict(self.mixer.state_shapes(), canon1=self.norm1.state_shape())
        if self.mlp is not None:
            out["canon2"] = self.norm2.state_shape()
        return out

    def checkpoint(self, prefix: str) -> dict:
        out = self.mixer.checkpoint(prefix + "mix.")
        out.update(self.norm1.checkpoint(prefix + "norm1", prefix + "canon1"))
        if self.mlp is not None:
            out.update(self.mlp.checkpoint(prefix + "mlp."))
            out.update(self.norm2.checkpoint(prefix + "norm2", prefix + "canon2"))
        return out

    def forward(self, x: torch.Tensor, layer_step) -> None:
        """Adds both sub-layers to the float32 stream ``x`` in place."""
        self.mixer(x, self.norm1(x, layer_step.state["canon1"], layer_step.batch), layer_step)
        if self.mlp is not None:
            self.mlp(x, self.norm2(x, layer_step.state["canon2"], layer_step.batch))


class VemedraForCausalLM(nn.Module):
    tp_size, tp_rank = 1, 0
    delegates_attention = False

    def __init__(self, cfg: VemedraConfig, *, device="cpu", dtype=torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise TypeError(f"Vemedra runs in bfloat16 or float32, not {dtype}")
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device(device)
        self.vocab_size = cfg.vocab
        self.register_buffer("embed", torch.zeros(cfg.vocab, cfg.width, dtype=dtype, device=device), persistent=False)
        self.register_buffer("head", torch.zeros(cfg.vocab, cfg.width, dtype=dtype, device=device), persistent=False)
        self.register_buffer("final_norm", torch.zeros(cfg.width, dtype=torch.float32, device=device), persistent=False)
        self.register_buffer("loop_step", torch.zeros(cfg.loop_times, cfg.width, dtype=torch.float32, device=device), persistent=False)
        self.layers = nn.ModuleList([VemedraLayer(cfg, spec, dtype=dtype, device=device) for spec in cfg.layers])
        self.runs = cfg.runs()

    # -------------------------------------------------------------- loading and caching
    def checkpoint_tensors(self) -> dict[str, torch.Tensor]:
        """Checkpoint name -> the view it is copied into (parts of merged weights among them)."""
        out = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        if self.cfg.loop_times > 0:
            out["loop.step"] = self.loop_step
        for i, layer in enumerate(self.layers):
            out.update(layer.checkpoint(f"l{i}."))
        return out

    def cache_layout(self) -> CacheLayout:
        return CacheLayout([self.layers[i].mixer.kv_spec() for i, _ in self.runs], [self.layers[i].state_shapes() for i, _ in self.runs])

    # -------------------------------------------------------------- one step
    def forward_step(self, batch: StepBatch, layer_step: Callable[[int], object], rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Runs the step's tokens from the caches and states that earlier steps left; returns the final norm of the
        given rows (all tokens if None)."""
        x = torch.empty(batch.num_tokens, self.cfg.width, dtype=torch.float32, device=self.device)
        first = self.runs[0][1] if self.runs else None  # the first layer may itself open a pass
        ops.stream_add(x, batch.tokens, self.embed, None if first is None else self.loop_step[first], False)
        for r, (i, t) in enumerate(self.runs):
            if t is not None and r > 0:
                # a later pass also adds the embedding output again
                ops.stream_add(x, batch.tokens if t > 0 else None, self.embed if t > 0 else None, self.loop_step[t], True)
            self.layers[i](x, layer_step(r))
        return ops.rmsnorm_rows(x, rows, self.final_norm, self.cfg.eps, self.dtype)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return ops.linear(hidden, self.head, torch.float32)

    @torch.no_grad()
    def greedy_tokens(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits(hidden).argmax(dim=-1)
