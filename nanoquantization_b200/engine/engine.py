"""A small serving engine: paged KV cache, recurrent-state pool, block manager, continuous-batching scheduler,
model runner with CUDA-graph decode.

The reference has none of this (its only execution is a full-sequence forward for a loss,
models/qwen3_quantized.py:326-341); it exists so that models are measured where they are used: prefill of batched
prompts (whole or in portions) and greedy decode steps over a cache.  A model states what it keeps per layer run
(``cache_layout()``) and runs one step on a ``StepBatch`` (``forward_step``).  For a model that delegates attention
(Qwen3) the engine supplies it: PyTorch's scaled_dot_product_attention per prompt at prefill; at decode flash_attn's
paged-KV kernel when that library loads on this GPU, else scaled_dot_product_attention over the gathered pages of
each sequence.  Other models bring kernels that read the cache and the states themselves.

Layout: per layer run two tensors ``[num_blocks, block_size, kv_heads, head_dim]``; a sequence owns a list of blocks;
``row = block * block_size + offset``.  Blocks that no later query can reach (every layer attends inside chunks) are
given back while the sequence runs.  A recurrent state is a row of ``[slots, ...]``; a sequence owns one slot.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Optional, Sequence as Seq

import torch
import torch.nn.functional as F

from .batch import CacheLayout, StepBatch


@dataclass
class Sequence:
    seq_id: int
    prompt: list[int]
    max_new_tokens: int
    output: list[int] = field(default_factory=list)
    blocks: list[int] = field(default_factory=list)
    prefilled: bool = False
    carried: list[int] = field(default_factory=list)  # tokens generated before a preemption (now part of the prompt)
    computed: int = 0  # tokens that the cache and the states hold
    slot: Optional[int] = None  # recurrent-state slot
    scheduled: int = 0  # tokens that the scheduler gave it in this step

    def __len__(self) -> int:
        return len(self.prompt) + len(self.output)

    @property
    def finished(self) -> bool:
        return len(self.output) >= self.max_new_tokens


class BlockManager:
    """Free-list allocator of KV-cache blocks."""

    def __init__(self, num_blocks: int, block_size: int):
        self.block_size = block_size
        self.free = deque(range(num_blocks))

    def blocks_needed(self, n_tokens: int) -> int:
        return -(-n_tokens // self.block_size)

    def can_allocate(self, n_tokens: int) -> bool:
        return self.blocks_needed(n_tokens) <= len(self.free)

    def ensure(self, seq: Sequence, n_tokens: int) -> bool:
        """Grow ``seq`` to hold ``n_tokens``; False (and no change) if the pool is exhausted."""
        need = self.blocks_needed(n_tokens) - len(seq.blocks)
        if need > len(self.free):
            return False
        for _ in range(max(need, 0)):
            seq.blocks.append(self.free.popleft())
        return True

    def reclaim(self, seq: Sequence, first_visible: int) -> None:
        """Give back the blocks that lie wholly before ``first_visible`` (their places in the list become -1)."""
        i = min(first_visible // self.block_size, len(seq.blocks)) - 1
        while i >= 0 and seq.blocks[i] >= 0:
            self.free.append(seq.blocks[i])
            seq.blocks[i] = -1
            i -= 1

    def release(self, seq: Sequence) -> None:
        self.free.extend(b for b in seq.blocks if b >= 0)
        seq.blocks = []


class PagedKVCache:
    """Keys and values of every layer run that keeps some (None for the others)."""

    def __init__(self, layout: CacheLayout, num_blocks, block_size, dtype, device):
        def pool(heads, dim):
            return torch.zeros(num_blocks, block_size, heads, dim, dtype=dtype, device=device)
        self.k = [None if s is None else pool(s.kv_heads, s.head_dim) for s in layout.kv]
        self.v = [None if s is None else pool(s.kv_heads, s.v_dim) for s in layout.kv]
        self.block_size = block_size

    def write(self, layer: int, slots: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> None:
        self.k[layer].view(-1, *k.shape[1:]).index_copy_(0, slots, k)
        self.v[layer].view(-1, *v.shape[1:]).index_copy_(0, slots, v)


class StatePool:
    """Recurrent states, float32: per layer run a dict of tensors ``[num_slots, ...]``.  A slot is not cleared when it
    changes hands: a step that starts a sequence (position 0) takes its states as zero."""

    def __init__(self, layout: CacheLayout, num_slots: int, device):
        self.states = [{k: torch.zeros(num_slots, *shape, dtype=torch.float32, device=device) for k, shape in run.items()}
                       for run in (layout.states or [{}] * len(layout.kv))]
        self.free = deque(range(num_slots - 1))  # the last one is for padding rows

    def ensure(self, seq: Sequence) -> bool:
        if seq.slot is None:
            if not self.free:
                return False
            seq.slot = self.free.popleft()
        return True

    def release(self, seq: Sequence) -> None:
        if seq.slot is not None:
            self.free.append(seq.slot)
            seq.slot = None


class LayerStep:
    """One layer run's share of a step: its caches and states, and the attention of models that delegate it
    (``attend(q, k, v)`` stores k and v and returns the output; ``stored``: the caller stored them already)."""

    def __init__(self, engine: "LLMEngine", run: int, batch: StepBatch, decode: bool):
        self.engine, self.batch, self.decode = engine, batch, decode
        self.k_cache, self.v_cache, self.state = engine.cache.k[run], engine.cache.v[run], engine.states.states[run]
        self.kv_target = (self.k_cache, self.v_cache, batch.rows)

    def __call__(self, q, k, v, stored=False):
        if not stored:
            self.k_cache.view(-1, *self.k_cache.shape[2:]).index_copy_(0, self.batch.rows, k)
            self.v_cache.view(-1, *self.v_cache.shape[2:]).index_copy_(0, self.batch.rows, v)
        return self._decode(q) if self.decode else self._prefill(q, k, v)

    def _gathered(self, table):
        """The pages of ``table [..., W]`` as ``[..., W * block_size, heads, dim]``."""
        kk, vv = self.k_cache[table.long()], self.v_cache[table.long()]
        return kk.flatten(-4, -3), vv.flatten(-4, -3)

    def _prefill(self, q, k, v):
        outs, o = [], 0
        for b, (n, start) in enumerate(zip(self.batch.lens, self.batch.starts)):
            qs, ks, vs, mask = q[o:o + n], k[o:o + n], v[o:o + n], None
            if start > 0:  # a later portion: the earlier ones' keys come from the cache
                kk, vv = self._gathered(self.batch.table[b])
                ks, vs = kk[:start + n], vv[:start + n]
                mask = torch.ones(n, start + n, dtype=torch.bool, device=q.device).tril(start)
            qs, ks, vs = (t.transpose(0, 1).unsqueeze(0) for t in (qs, ks, vs))
            outs.append(F.scaled_dot_product_attention(qs, ks, vs, attn_mask=mask, is_causal=mask is None,
                                                       enable_gqa=qs.shape[1] != ks.shape[1])[0].transpose(0, 1))
            o += n
        return torch.cat(outs, dim=0)

    def _decode(self, q):
        if self.engine.paged_attention is not None:
            return self.engine.paged_attention(q.unsqueeze(1), self.k_cache, self.v_cache, cache_seqlens=self.batch.ctx,
                                               block_table=self.batch.table, causal=True).squeeze(1)
        kk, vv = self._gathered(self.batch.table)
        mask = torch.arange(kk.shape[1], device=q.device)[None, :] < self.batch.ctx[:, None]          # [B, S]
        o = F.scaled_dot_product_attention(q.unsqueeze(2), kk.transpose(1, 2), vv.transpose(1, 2),
                                           attn_mask=mask[:, None, None, :], enable_gqa=q.shape[1] != kk.shape[2])
        return o.squeeze(2)


class Scheduler:
    """Prefill has priority: waiting prompts are admitted while blocks and the token budget last;
    otherwise every running sequence decodes one token.  A sequence that cannot grow is preempted
    (its blocks are released and it returns to the waiting queue to be prefilled again).

    ``portion``: a prefill step takes so many tokens at most and a prompt that does not fit into what is left of
    them is cut; it stays in the waiting queue, with what it holds, until its last portion has run."""

    def __init__(self, blocks: BlockManager, max_batch: int, max_prefill_tokens: int, portion: Optional[int] = None,
                 states: Optional[StatePool] = None):
        self.blocks, self.max_batch, self.max_prefill_tokens = blocks, max_batch, max_prefill_tokens
        self.portion, self.states = portion, states
        self.waiting: deque[Sequence] = deque()
        self.running: list[Sequence] = []

    def add(self, seq: Sequence) -> None:
        self.waiting.append(seq)

    def _admit(self, s: Sequence, n_tokens: int) -> bool:
        if self.states is not None and not self.states.ensure(s):
            return False
        return self.blocks.ensure(s, n_tokens)

    def release(self, s: Sequence) -> None:
        self.blocks.release(s)
        if self.states is not None:
            self.states.release(s)
        s.computed = 0

    def step(self) -> tuple[str, list[Sequence]]:
        kind, batch = self._step()
        if not batch and not self.running:
            # nothing can move: sequences that wait in the middle of their prompts may hold what the head needs
            for s in list(self.waiting)[:0:-1]:
                if s.blocks:
                    self.release(s)
                    return self.step()
        return kind, batch

    def _step(self) -> tuple[str, list[Sequence]]:
        batch, tokens = [], 0
        for s in list(self.waiting):
            if len(self.running) + len(batch) >= self.max_batch:
                break
            n = len(s) - s.computed
            if self.portion is not None:
                n = min(n, self.portion - tokens)
                if n <= 0:
                    break
            elif tokens + n > self.max_prefill_tokens and batch:
                break
            end = s.computed + n
            if not self._admit(s, end + 1 if end == len(s) else end):
                break
            s.scheduled = n
            batch.append(s)
            tokens += n
        if batch:
            for s in batch:
                if s.computed + s.scheduled == len(s):
                    self.waiting.remove(s)
            return "prefill", batch
        ready = []
        i = 0
        while i < len(self.running):
            s = self.running[i]
            if self.blocks.ensure(s, len(s) + 1):
                ready.append(s)
                i += 1
                continue
            # no block left for s to grow into: preempt the youngest running sequence and try again
            victim = self.running.pop()
            self.release(victim)
            if victim in ready:
                ready.remove(victim)
            victim.carried += victim.output
            victim.max_new_tokens -= len(victim.output)
            victim.prompt, victim.output, victim.prefilled = victim.prompt + victim.output, [], False
            self.waiting.appendleft(victim)
        return "decode", ready

    def finish_step(self, kind: str, batch: list[Sequence]) -> list[Sequence]:
        """``batch``: the sequences that got a token (a prompt whose portions have not all run got none)."""
        done = []
        if kind == "prefill":
            self.running.extend(batch)
        for s in batch:
            if s.finished:
                done.append(s)
                self.running.remove(s)
                self.release(s)
        return done


class LLMEngine:
    def __init__(self, model, num_blocks: int, block_size: int = 256, max_batch: int = 64,
                 max_prefill_tokens: int = 16384, use_cuda_graph: bool = True, prefill_portion: Optional[int] = None):
        self.model = model
        self.device, self.dtype = model.device, model.dtype
        self.layout = model.cache_layout()
        self.block_size = block_size
        # one block and one slot more than are handed out: padding rows of a bucketed decode batch write there
        self.cache = PagedKVCache(self.layout, num_blocks + 1, block_size, self.dtype, self.device)
        self.states = StatePool(self.layout, max_batch + 1, self.device)
        self.scratch_block, self.scratch_slot = num_blocks, max_batch
        self.blocks = BlockManager(num_blocks, block_size)
        self.scheduler = Scheduler(self.blocks, max_batch, max_prefill_tokens, prefill_portion, self.states)
        self.use_cuda_graph = use_cuda_graph
        self.paged_attention = self._probe_flash_attn() if model.delegates_attention and block_size % 256 == 0 else None
        self._graphs: dict[tuple[int, int], tuple] = {}
        self._warm_stream = None  # one side stream for every graph warm-up (scratch buffers are kept per stream)
        self._next_id = 0
        self.max_tokens_per_sequence = num_blocks * block_size

    # ------------------------------------------------------------------ attention
    def _probe_flash_attn(self):
        """flash_attn's paged decode kernel if this build of it runs on this GPU, else None (the
        fallback gathers the pages and calls scaled_dot_product_attention)."""
        try:
            from flash_attn import flash_attn_with_kvcache
            heads = self.model.model.layers[0].self_attn.num_heads
            q = torch.zeros(1, 1, heads, self.layout.kv[0].head_dim, dtype=self.dtype, device=self.device)
            bt = torch.zeros(1, 1, dtype=torch.int32, device=self.device)
            ln = torch.ones(1, dtype=torch.int32, device=self.device)
            flash_attn_with_kvcache(q, self.cache.k[0], self.cache.v[0], cache_seqlens=ln, block_table=bt, causal=True)
            torch.cuda.synchronize()
            return flash_attn_with_kvcache
        except Exception:  # not built for this architecture, or not importable
            return None

    # --------------------------------------------------------------------- steps
    def _forward(self, batch: StepBatch, decode: bool, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return self.model.forward_step(batch, lambda run: LayerStep(self, run, batch, decode), rows)

    def _hold(self, s: Sequence, n_tokens: int) -> None:
        if not self.states.ensure(s) or not self.blocks.ensure(s, n_tokens):
            raise RuntimeError(f"the cache cannot hold {n_tokens} tokens of sequence {s.seq_id}")

    def _advance(self, s: Sequence, computed: int) -> None:
        s.computed = computed
        self.blocks.reclaim(s, self.layout.visible_from(computed))

    def _run_portions(self, batch: list[Sequence], counts: list[int], rows: Optional[list[int]] = None) -> torch.Tensor:
        """The next ``counts[i]`` tokens of each sequence, from what earlier steps left; the final hidden states of
        the given rows of the step (default: each sequence's last)."""
        tokens = [(s.prompt + s.output)[s.computed:s.computed + n] for s, n in zip(batch, counts)]
        for s in batch:
            self.states.ensure(s)
        width = max(1, max(len(s.blocks) for s in batch))
        host = StepBatch.host(tokens, [s.computed for s in batch], [s.blocks for s in batch],
                              [self.scratch_slot if s.slot is None else s.slot for s in batch], width, self.block_size)
        if rows is None:
            rows = [e - 1 for e in host.cu.tolist()[1:]]
        h = self._forward(host.to(self.device), False, torch.tensor(rows, dtype=torch.long, device=self.device))
        for s, n in zip(batch, counts):
            self._advance(s, s.computed + n)
        return h

    @torch.no_grad()
    def _prefill(self, batch: list[Sequence], counts: Optional[list[int]] = None) -> torch.Tensor:
        if counts is None:  # whole prompts
            for s in batch:
                s.computed = 0
            counts = [len(s) for s in batch]
        return self.model.greedy_tokens(self._run_portions(batch, counts))

    def _decode_inputs(self, batch: list[Sequence], width: int, rows: Optional[int] = None) -> StepBatch:
        """Host side of one decode step.  ``rows`` > len(batch) pads the batch: a padding row is token 0 at
        position 0 of a one-token sequence that lives in the scratch block and slot."""
        for s in batch:
            self.states.ensure(s)
        pad = (len(batch) if rows is None else rows) - len(batch)
        return StepBatch.host([[(s.output or s.prompt)[-1]] for s in batch] + [[0]] * pad, [len(s) - 1 for s in batch] + [0] * pad,
                              [s.blocks for s in batch] + [[self.scratch_block]] * pad,
                              [self.scratch_slot if s.slot is None else s.slot for s in batch] + [self.scratch_slot] * pad,
                              width, self.block_size)

    def _decode_forward(self, batch: StepBatch):
        h = self._forward(batch, True)
        return h, self.model.greedy_tokens(h)

    @torch.no_grad()
    def _decode_hidden(self, batch: list[Sequence]):
        """One token of every sequence: final hidden states and greedy choices."""
        B = len(batch)
        width = max(1, max(len(s.blocks) for s in batch))
        if not self.use_cuda_graph:
            h, out = self._decode_forward(self._decode_inputs(batch, width).to(self.device))
        else:
            # one graph per (batch bucket, block-table width): batches are padded up to a power of two, so that
            # continuous batching replays a few dozen graphs.  For the engine's own attention the block table keeps
            # its exact width, by which that kernel sizes its KV splits (a table padded from 9 to 16 blocks cost
            # 18 % of a step); kernels that look up their own pages take a width rounded up as well
            rows = 1 << (B - 1).bit_length()
            if not self.model.delegates_attention:
                width = 1 << (width - 1).bit_length()
            host = self._decode_inputs(batch, width, rows)
            key = (rows, width)
            if key not in self._graphs:
                self._graphs[key] = self._capture(host)
            graph, static, h, out = self._graphs[key]
            static.copy_(host)
            graph.replay()
            h, out = h[:B], out[:B]
        for s in batch:
            self._advance(s, len(s))
        return h, out

    def _capture(self, host: StepBatch):
        # the warm-up outside the capture runs on padding: every row in the scratch block and slot, so that no
        # sequence's state advances by it
        n, width = host.batch, host.width
        static = StepBatch.host([[0]] * n, [0] * n, [[self.scratch_block]] * n, [self.scratch_slot] * n, width, self.block_size).to(self.device)
        if self._warm_stream is None:
            self._warm_stream = torch.cuda.Stream()
        side = self._warm_stream
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            self._decode_forward(static)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            h, out = self._decode_forward(static)
        return graph, static, h, out

    def _decode(self, batch: list[Sequence]) -> torch.Tensor:
        return self._decode_hidden(batch)[1]

    @torch.no_grad()
    def extend(self, entries: Seq[tuple[Sequence, Seq[int], Seq[int]]]) -> list[torch.Tensor]:
        """One step on tokens that are given, not chosen: ``(sequence, next tokens, wanted places among them)`` per
        entry; returns the wanted logits, ``[places, vocab]`` each.  Single tokens that continue their sequences
        take the decode path, anything else the prefill path, as in generation."""
        batch, counts = [s for s, _, _ in entries], [len(t) for _, t, _ in entries]
        for s, tokens, _ in entries:
            s.prompt.extend(tokens)
            self._hold(s, len(s))
        if all(n == 1 and s.computed > 0 for s, n in zip(batch, counts)):
            h = self._decode_hidden(batch)[0]
            return [self.model.logits(h[i:i + 1]) if len(want) else None for i, (_, _, want) in enumerate(entries)]
        rows, o = [], 0
        for (_, _, want), n in zip(entries, counts):
            rows += [o + w for w in want]
            o += n
        h = self._run_portions(batch, counts, rows)
        out, o = [], 0
        for _, _, want in entries:
            out.append(self.model.logits(h[o:o + len(want)]) if len(want) else None)
            o += len(want)
        return out

    def drop(self, s: Sequence) -> None:
        """Give back what a sequence holds."""
        self.scheduler.release(s)

    # ----------------------------------------------------------------------- API
    def add_request(self, prompt: Seq[int], max_new_tokens: int) -> int:
        if len(prompt) + 1 > self.max_tokens_per_sequence:
            raise ValueError(f"a prompt of {len(prompt)} tokens can never be admitted: the KV cache holds "
                             f"{self.max_tokens_per_sequence} tokens in all")
        sid = self._next_id
        self._next_id += 1
        self.scheduler.add(Sequence(sid, list(prompt), max_new_tokens))
        return sid

    def step(self) -> list[Sequence]:
        kind, batch = self.scheduler.step()
        if not batch:
            if self.scheduler.waiting and not self.scheduler.running:
                raise RuntimeError("the head of the waiting queue cannot be admitted although nothing is running "
                                   "(the KV cache is too small for it)")
            return []
        if kind == "prefill":
            new = self._prefill(batch, [s.scheduled for s in batch]).tolist()
        else:
            new = self._decode(batch).tolist()
        self._check_device_status()
        complete = [s for s in batch if s.computed == len(s)]
        for s, t in zip(batch, new):
            if s.computed == len(s):  # a prompt whose last portion has not run yet gets no token
                s.output.append(int(t))
                s.prefilled = True
        return self.scheduler.finish_step(kind, complete)

    def _check_device_status(self) -> None:
        """After the step's results reached the host: raise if a bounded device-side wait gave up during it
        (a peer that never arrived at an all-reduce, a pipeline barrier inside a GEMM).  Such a kernel
        returns without writing its output, so the step's tokens would be garbage."""
        from .. import _lib
        comm = getattr(self.model, "tp_comm", None)
        if comm is not None:
            comm.check()
        if self.device.type == "cuda":
            _lib.check_workspaces()
            _lib.check_mixer_status()

    def generate(self, prompts: Seq[Seq[int]], max_new_tokens) -> list[list[int]]:
        if isinstance(max_new_tokens, int):
            max_new_tokens = [max_new_tokens] * len(prompts)
        ids = [self.add_request(p, n) for p, n in zip(prompts, max_new_tokens)]
        results: dict[int, list[int]] = {}
        while self.scheduler.waiting or self.scheduler.running:
            for s in self.step():
                results[s.seq_id] = s.carried + s.output
        return [results[i] for i in ids]
