"""What a model's step works on: the flattened tokens of several sequences, where each sequence stands, which K/V
blocks and which recurrent-state slot it owns.

``CacheLayout`` is a model's statement of what it keeps per layer run: keys and values in the paged cache
(``KVSpec``), recurrent states in the state pool (shapes), either, both or none."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field
from typing import Optional, Sequence as Seq

import numpy as np
import torch

from .. import _lib


@dataclass(frozen=True)
class KVSpec:
    """``chunk``: no query looks behind its own chunk of so many positions (None: it may see everything)."""
    kv_heads: int
    head_dim: int
    v_dim: int
    chunk: Optional[int] = None


@dataclass
class CacheLayout:
    kv: list[Optional[KVSpec]]
    states: list[dict[str, tuple]] = field(default_factory=list)

    @property
    def recurrent(self) -> bool:
        return any(self.states)

    def visible_from(self, position: int) -> int:
        """The first position whose keys and values a query at ``position`` or later can still reach."""
        floor = position
        for s in self.kv:
            if s is not None:
                floor = min(floor, position // s.chunk * s.chunk if s.chunk else 0)
        return floor


class StepBatch:
    """Two flat integer buffers (one copy each to the device) and named views of them.

    int64: ``tokens``, ``positions``, ``rows`` (cache row of each token), each [T].
    int32: ``cu`` [B + 1] token bounds, ``pos0`` [B] first position, ``ctx`` [B] context length after the step,
    ``slot`` [B] state slot, ``table`` [B, W] K/V blocks."""

    def __init__(self, i64: torch.Tensor, i32: torch.Tensor, lens: Seq[int], starts: Seq[int], width: int, block_size: int):
        T, B = sum(lens), len(lens)
        self.i64, self.i32, self.lens, self.starts = i64, i32, list(lens), list(starts)
        self.num_tokens, self.batch, self.width, self.block_size = T, B, width, block_size
        self.max_len = max(lens) if lens else 0
        self.tokens, self.positions, self.rows = i64[:T], i64[T:2 * T], i64[2 * T:3 * T]
        self.cu, self.pos0, self.ctx, self.slot = i32[:B + 1], i32[B + 1:2 * B + 1], i32[2 * B + 1:3 * B + 1], i32[3 * B + 1:4 * B + 1]
        self.table = i32[4 * B + 1:].view(B, width)
        self.desc = _lib.StepDesc(self.cu.data_ptr(), self.pos0.data_ptr(), self.slot.data_ptr(), self.table.data_ptr(), B, T,
                                  self.max_len, width, block_size)

    @classmethod
    def host(cls, tokens: Seq[Seq[int]], starts: Seq[int], blocks: Seq[Seq[int]], slots: Seq[int], width: int, block_size: int) -> "StepBatch":
        """Sequence b brings ``tokens[b]``, the first at position ``starts[b]``; a block of -1 is one it no longer holds."""
        lens = [len(t) for t in tokens]
        T, B = sum(lens), len(lens)
        i64, i32 = np.empty(3 * T, np.int64), np.zeros(4 * B + 1 + B * width, np.int32)
        i32[1:B + 1] = np.cumsum(lens)
        i32[B + 1:2 * B + 1] = starts
        i32[2 * B + 1:3 * B + 1] = np.asarray(starts) + np.asarray(lens)
        i32[3 * B + 1:4 * B + 1] = slots
        table = i32[4 * B + 1:].reshape(B, width)
        o = 0
        for b, (toks, n, p) in enumerate(zip(tokens, lens, starts)):
            table[b, :len(blocks[b])] = np.maximum(np.asarray(blocks[b], np.int32), 0) if blocks[b] else 0
            pos = np.arange(p, p + n)
            i64[o:o + n] = toks
            i64[T + o:T + o + n] = pos
            i64[2 * T + o:2 * T + o + n] = table[b, pos // block_size].astype(np.int64) * block_size + pos % block_size
            o += n
        return cls(torch.from_numpy(i64), torch.from_numpy(i32), lens, starts, width, block_size)

    def to(self, device) -> "StepBatch":
        return StepBatch(self.i64.to(device), self.i32.to(device), self.lens, self.starts, self.width, self.block_size)

    def copy_(self, other: "StepBatch") -> None:
        """Take over another batch of the same shape (the inputs of a captured graph)."""
        self.i64.copy_(other.i64, non_blocking=True)
        self.i32.copy_(other.i32, non_blocking=True)
