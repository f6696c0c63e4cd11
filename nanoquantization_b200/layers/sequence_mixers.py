"""Sub-layers of decoders that mix tokens by other means than plain attention, over the kernels of ``mixers.py``.

A mixer owns two merged weights, ``w_in [rows, width]`` (everything that reads the sub-layer's input, one product)
and ``w_out [width, columns]`` (everything that is added to the residual stream, one product), and says what it
keeps per sequence: ``kv_spec()`` for the paged cache, ``state_shapes()`` for the recurrent-state pool.  ``mix(proj,
act, layer_step)`` turns the input product into the operand of the output product.  ``checkpoint(prefix)`` names
the views of the merged weights that checkpoint tensors are copied into.

Mixers that can stand side by side (``AttentionMixer``, ``RetentionMixer``) take their columns of ``proj`` and
``act`` as offsets, so that ``ParallelMixer`` runs both on one product each; their output scale goes into the
kernel that writes ``act``."""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import _lib
from ..engine.batch import KVSpec
from . import mixers as ops
from . import moe


def _buffer(module: nn.Module, name: str, *shape, dtype, device) -> torch.Tensor:
    module.register_buffer(name, torch.zeros(*shape, dtype=dtype, device=device), persistent=False)
    return getattr(module, name)


def _inverse_frequencies(base, dims, device):
    i = torch.arange(dims // 2, dtype=torch.float64)
    return (float(base) ** (-2.0 * i / max(dims, 1))).float().to(device)


class AttentionMixer(nn.Module):
    """Grouped-query attention inside chunks of the sequence, partial rotary embedding, capped scores, a sink per head."""

    def __init__(self, *, heads, kv_heads, dim, vdim, chunk, rot_base, rot_dims, scale, softcap, out_scale=1.0, device="cpu"):
        super().__init__()
        if heads % kv_heads != 0 or rot_dims % 2 != 0 or not 0 <= rot_dims <= dim:
            raise ValueError(f"attention: {heads} heads over {kv_heads} key/value heads, {rot_dims} of {dim} dimensions rotated")
        if chunk < 1 or softcap <= 0:
            raise ValueError(f"attention: chunk {chunk} and softcap {softcap} must be positive")
        self.heads, self.kv_heads, self.dim, self.vdim, self.chunk = heads, kv_heads, dim, vdim, chunk
        self.scale, self.softcap, self.out_scale = float(scale), float(softcap), float(out_scale)
        self.in_parts = [("q", heads * dim), ("k", kv_heads * dim), ("v", kv_heads * vdim)]
        self.out_columns = heads * vdim
        _buffer(self, "sink", heads, dtype=torch.float32, device=device)
        self.register_buffer("inv_freq", _inverse_frequencies(rot_base, rot_dims, device), persistent=False)

    def kv_spec(self):
        return KVSpec(self.kv_heads, self.dim, self.vdim, self.chunk)

    def state_shapes(self):
        return {}

    def checkpoint(self, prefix):
        return {prefix + "sink": self.sink}

    def desc(self) -> _lib.AttentionDesc:
        return _lib.AttentionDesc(self.heads, self.kv_heads, self.dim, self.vdim, self.chunk, self.scale, self.softcap,
                                  self.sink.data_ptr(), self.out_scale, None, None, 0)

    def rope_desc(self) -> _lib.RopeDesc:
        return _lib.RopeDesc(self.heads, self.kv_heads, self.dim, self.vdim, 2 * self.inv_freq.numel(), 0, self.inv_freq.data_ptr(), None, None, 0.0)

    def value_column(self, col):
        return col + (self.heads + self.kv_heads) * self.dim

    def mix(self, proj, col, act, act_col, layer_step):
        q_off, k_off, v_off = col, col + self.heads * self.dim, col + (self.heads + self.kv_heads) * self.dim
        ops.rope_store(proj, layer_step.k_cache, layer_step.v_cache, self.inv_freq, layer_step.batch, q_off, k_off, v_off, self.heads)
        ops.chunk_attention(proj[:, q_off:k_off], layer_step.k_cache, layer_step.v_cache, act[:, act_col:act_col + self.out_columns],
                            self.desc(), layer_step.batch)


class SigmoidAttentionMixer(nn.Module):
    """Grouped-query attention whose weights are sigmoids of the scores (plus a number per head), not normalised over the
    keys.  Queries and keys are RMS-normed per head and partially rotated; the values are the keys as projected."""

    def __init__(self, *, heads, kv_heads, dim, rot_base, rot_dims, interleaved, scale, eps, out_scale=1.0, device="cpu"):
        super().__init__()
        if heads % kv_heads != 0 or rot_dims % 2 != 0 or not 0 <= rot_dims <= dim:
            raise ValueError(f"attention: {heads} heads over {kv_heads} key/value heads, {rot_dims} of {dim} dimensions rotated")
        self.heads, self.kv_heads, self.dim, self.vdim, self.rot = heads, kv_heads, dim, dim, rot_dims
        self.scale, self.eps, self.out_scale, self.interleaved = float(scale), float(eps), float(out_scale), bool(interleaved)
        self.in_parts = [("q", heads * dim), ("k", kv_heads * dim)]
        self.out_columns = heads * dim
        for name, n in (("q_norm", dim), ("k_norm", dim), ("temp", heads), ("bias", heads)):
            _buffer(self, name, n, dtype=torch.float32, device=device)
        self.register_buffer("inv_freq", _inverse_frequencies(rot_base, rot_dims, device), persistent=False)

    def kv_spec(self):
        return KVSpec(self.kv_heads, self.dim, self.vdim)

    def state_shapes(self):
        return {}

    def checkpoint(self, prefix):
        return {prefix + "q.norm": self.q_norm, prefix + "k.norm": self.k_norm, prefix + "temp": self.temp, prefix + "pb": self.bias}

    def desc(self) -> _lib.AttentionDesc:
        return _lib.AttentionDesc(self.heads, self.kv_heads, self.dim, self.vdim, 0, self.scale, 0.0, None, self.out_scale, self.temp.data_ptr(),
                                  self.bias.data_ptr(), 1)

    def rope_desc(self) -> _lib.RopeDesc:
        return _lib.RopeDesc(self.heads, self.kv_heads, self.dim, self.vdim, self.rot, int(self.interleaved), self.inv_freq.data_ptr(),
                             self.q_norm.data_ptr(), self.k_norm.data_ptr(), self.eps)

    def value_column(self, col):
        return col + self.heads * self.dim

    def mix(self, proj, col, act, act_col, layer_step):
        q_off, k_off = col, col + self.heads * self.dim
        ops.norm_rope(proj, layer_step.k_cache, layer_step.v_cache, self.rope_desc(), layer_step.batch, q_off, k_off, k_off)
        ops.chunk_attention(proj[:, q_off:k_off], layer_step.k_cache, layer_step.v_cache, act[:, act_col:act_col + self.out_columns],
                            self.desc(), layer_step.batch)


class RetentionMixer(nn.Module):
    """Linear attention with one fixed decay per head, queries and keys rotated where ``rot_dims`` says so (pairs i, i +
    rot_dims / 2); each head's output is RMS-normalised and gated."""

    state_name = "retention"

    def __init__(self, *, heads, dim, vdim, decay, eps, out_scale=1.0, rot_base=1.0, rot_dims=0, device="cpu"):
        super().__init__()
        if rot_dims % 2 != 0 or not 0 <= rot_dims <= dim:
            raise ValueError(f"retention: {rot_dims} of {dim} dimensions rotated")
        if len(decay) != heads:
            raise ValueError(f"retention: {len(decay)} decays for {heads} heads")
        self.heads, self.dim, self.vdim, self.eps, self.out_scale = heads, dim, vdim, float(eps), float(out_scale)
        self.in_parts = [("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim)]
        self.out_columns = heads * vdim
        self.rot = rot_dims
        self.register_buffer("decay", torch.tensor(decay, dtype=torch.float64).float().to(device), persistent=False)
        self.register_buffer("inv_freq", _inverse_frequencies(rot_base, rot_dims, device), persistent=False)

    def kv_spec(self):
        return None

    def state_shapes(self):
        return {self.state_name: (self.heads, self.dim, self.vdim)}

    def checkpoint(self, prefix):
        return {}

    def desc(self) -> _lib.RetentionDesc:
        return _lib.RetentionDesc(self.heads, self.dim, self.vdim, self.eps, self.out_scale, self.decay.data_ptr(), None,
                                  self.inv_freq.data_ptr(), self.rot)

    def rope_desc(self) -> _lib.RopeDesc:
        return _lib.RopeDesc(self.heads, self.heads, self.dim, self.vdim, self.rot, 0, self.inv_freq.data_ptr(), None, None, 0.0)

    def mix(self, proj, col, act, act_col, layer_step):
        if self.rot > 0:
            ops.norm_rope(proj, None, None, self.rope_desc(), layer_step.batch, col, col + self.heads * self.dim, 0)
        ops.retention_gated(proj, col, self.desc(), self.decay, layer_step.state["retention"], act, act_col, layer_step.batch)


class GatedLinearMixer(nn.Module):
    """Gated linear attention: a decay per key channel and token, sigmoid(z)^(1 / tau) with z a low-rank projection of the
    input; each head's output is RMS-normalised with a weight and gated."""

    state_name = "gla"

    def __init__(self, *, heads, dim, vdim, rank, tau, eps, out_scale=1.0, dtype=torch.bfloat16, device="cpu"):
        super().__init__()
        if tau <= 0:
            raise ValueError(f"gated linear attention: tau {tau} must be positive")
        self.heads, self.dim, self.vdim, self.rank = heads, dim, vdim, rank
        self.tau, self.eps, self.out_scale = float(tau), float(eps), float(out_scale)
        self.in_parts = [("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim), ("a1", rank)]
        self.out_columns = heads * vdim
        _buffer(self, "a2", heads * dim, rank, dtype=dtype, device=device)
        _buffer(self, "a2_bias", heads * dim, dtype=torch.float32, device=device)
        _buffer(self, "norm", vdim, dtype=torch.float32, device=device)

    def kv_spec(self):
        return None

    def state_shapes(self):
        return {self.state_name: (self.heads, self.dim, self.vdim)}

    def desc(self) -> _lib.RetentionDesc:
        return _lib.RetentionDesc(self.heads, self.dim, self.vdim, self.eps, self.out_scale, None, self.norm.data_ptr(), None, 0, self.rank,
                                  self.tau, self.a2.data_ptr(), self.a2_bias.data_ptr())

    def checkpoint(self, prefix):
        return {prefix + "a2": self.a2, prefix + "a2.b": self.a2_bias, prefix + "norm": self.norm}

    def mix(self, proj, col, act, act_col, layer_step):
        ops.gla_gated(proj, col, self, layer_step.state["gla"], act, act_col, layer_step.batch)


class ParallelMixer(nn.Module):
    """Mixers side by side on the same input, their (scaled) outputs summed: one merged product in, one out.  ``beta``
    scales the stream that the sum is added to; ``prefixes`` names a part's tensors where they do not start with its name."""

    def __init__(self, width: int, parts: dict, *, dtype, device="cpu", beta=1.0, prefixes=None):
        super().__init__()
        self.parts, self.beta, self.prefixes = nn.ModuleDict(parts), float(beta), prefixes or {k: k + "." for k in parts}
        # rows of zeros fill up to a multiple of 8: rows of the product then start on 16-byte boundaries
        self.rows = -(-sum(n for m in parts.values() for _, n in m.in_parts) // 8) * 8
        self.columns = sum(m.out_columns for m in parts.values())
        _buffer(self, "w_in", self.rows, width, dtype=dtype, device=device)
        _buffer(self, "w_out", width, self.columns, dtype=dtype, device=device)
        # (mixer, first row of its projections, first column of its output), for the one-launch decode step
        self._attention = self._retention = None
        self._at_once = None
        row = col = 0
        for m in parts.values():
            if isinstance(m, (AttentionMixer, SigmoidAttentionMixer)):
                self._attention = (m, row, col)
            elif isinstance(m, (RetentionMixer, GatedLinearMixer)):
                self._retention = (m, row, col)
            row += sum(n for _, n in m.in_parts)
            col += m.out_columns

    def _decodes_at_once(self, h, batch) -> bool:
        if batch.max_len != 1 or h.dtype != torch.bfloat16:
            return False
        if self._at_once is None:
            self._at_once = (len(self.parts) == (self._attention is not None) + (self._retention is not None)
                             and ops.mixer_decode_supported(self._attention and self._attention[0].desc(),
                                                            self._retention and self._retention[0].desc()))
        return self._at_once

    def kv_spec(self):
        specs = [s for s in (m.kv_spec() for m in self.parts.values()) if s is not None]
        if len(specs) > 1:
            raise ValueError("one mixer of a layer keeps keys and values at most")
        return specs[0] if specs else None

    def state_shapes(self):
        return {k: v for m in self.parts.values() for k, v in m.state_shapes().items()}

    def checkpoint(self, prefix):
        out, row, col = {}, 0, 0
        for name, m in self.parts.items():
            p = prefix + self.prefixes[name]
            for part, n in m.in_parts:
                out[p + part] = self.w_in[row:row + n]
                row += n
            out[p + "o"] = self.w_out[:, col:col + m.out_columns]
            col += m.out_columns
            out.update(m.checkpoint(p))
        return out

    def mix(self, proj, act, layer_step):
        """The input product -> the operand of the output product; a decode step in one launch where its kernel takes the sizes."""
        if self._decodes_at_once(proj, layer_step.batch):
            att, ret = self._attention, self._retention
            ops.mixer_decode(proj, act, att and (att[0].desc(), att[0].rope_desc(), att[1], att[0].value_column(att[1]), att[2], layer_step.k_cache,
                                                 layer_step.v_cache),
                             ret and (ret[0].desc(), ret[1], ret[2], layer_step.state[ret[0].state_name]), layer_step.batch)
            return
        row = col = 0
        for m in self.parts.values():
            m.mix(proj, row, act, col, layer_step)
            row += sum(n for _, n in m.in_parts)
            col += m.out_columns

    def forward(self, x, h, layer_step):
        """``x = beta * x + mixer(h)`` on the float32 stream."""
        proj = ops.linear(h, self.w_in)
        act = torch.empty(h.shape[0], self.columns, dtype=h.dtype, device=h.device)
        self.mix(proj, act, layer_step)
        ops.linear_residual_(x, act, self.w_out, self.beta)


class MinGRUMixer(nn.Module):
    """A gated element-wise recurrence whose gates read the current token only."""

    def __init__(self, width: int, size: int, *, dtype, device="cpu"):
        super().__init__()
        self.size = size
        _buffer(self, "w_in", 3 * size, width, dtype=dtype, device=device)
        _buffer(self, "w_out", width, size, dtype=dtype, device=device)
        _buffer(self, "z_bias", size, dtype=torch.float32, device=device)
        _buffer(self, "x_bias", size, dtype=torch.float32, device=device)

    def kv_spec(self):
        return None

    def state_shapes(self):
        return {"mingru": (self.size,)}

    def checkpoint(self, prefix):
        n = self.size
        return {prefix + "z": self.w_in[:n], prefix + "x": self.w_in[n:2 * n], prefix + "g": self.w_in[2 * n:], prefix + "o": self.w_out,
                prefix + "z.b": self.z_bias, prefix + "x.b": self.x_bias}

    def forward(self, x, h, layer_step):
        if layer_step.batch.max_len == 1 and ops.decode_sized(h, self.w_in):
            y = ops.dense_mingru(h, self.w_in, self.z_bias, self.x_bias, layer_step.state["mingru"], layer_step.batch)
            ops.linear_residual_(x, y, self.w_out)
            return
        proj = ops.linear(h, self.w_in)
        y = ops.mingru(proj, self.size, self.z_bias, self.x_bias, layer_step.state["mingru"], layer_step.batch)
        ops.linear_residual_(x, y, self.w_out)


class ClampedGLU(nn.Module):
    """Feed-forward ``down(g sigmoid(1.702 g) (u + 1))`` with g and u clamped to a limit."""

    def __init__(self, width: int, ff: int, limit: float, *, dtype, device="cpu"):
        super().__init__()
        self.ff, self.limit = ff, float(limit)
        _buffer(self, "w_in", 2 * ff, width, dtype=dtype, device=device)
        _buffer(self, "w_out", width, ff, dtype=dtype, device=device)

    def checkpoint(self, prefix):
        return {prefix + "gate": self.w_in[:self.ff], prefix + "up": self.w_in[self.ff:], prefix + "down": self.w_out}

    def forward(self, x, h):
        if ops.decode_sized(h, self.w_in):
            ops.linear_residual_(x, ops.dense_glu(h, self.w_in, self.limit), self.w_out)
            return
        ops.linear_residual_(x, ops.clamped_glu(ops.linear(h, self.w_in), self.limit), self.w_out)


class RoutedExperts(nn.Module):
    """Feed-forward of many small experts ``down(gelu(up h))``, of which each token uses ``top``, chosen by sigmoid scores
    plus a correction among the best groups of neighbouring experts."""

    def __init__(self, width: int, ff: int, *, experts, top, groups, keep, scale, dtype, device="cpu"):
        super().__init__()
        if groups < 1 or experts % groups != 0 or not 1 <= keep <= groups or not 1 <= top <= keep * (experts // groups):
            raise ValueError(f"experts: {top} of {experts} from {keep} of {groups} groups")
        self.experts, self.top, self.groups, self.keep, self.scale = experts, top, groups, keep, float(scale)
        _buffer(self, "router", experts, width, dtype=dtype, device=device)
        _buffer(self, "correction", experts, dtype=torch.float32, device=device)
        _buffer(self, "up", experts, ff, width, dtype=dtype, device=device)
        _buffer(self, "down", experts, width, ff, dtype=dtype, device=device)

    def checkpoint(self, prefix):
        out = {prefix + "router": self.router, prefix + "correction": self.correction}
        for e in range(self.experts):
            out.update({f"{prefix}e{e}.up": self.up[e], f"{prefix}e{e}.down": self.down[e]})
        return out

    def router_desc(self) -> _lib.RouterDesc:
        return _lib.RouterDesc(self.experts, self.top, self.groups, self.keep, self.scale, self.correction.data_ptr())

    def forward(self, h):
        """The weighted outputs of every token's experts, ``[tokens, top, width]``; the caller adds them up."""
        plan = moe.route(ops.linear(h, self.router, torch.float32), self.router_desc())
        return moe.experts_down(moe.experts_up(h, self.up, plan), self.down, plan)


class GroupNorm(nn.Module):
    """RMS norm in groups after the residual sum: ``x = norm(alpha x + y)`` on the stream, and its rounding for what reads it."""

    def __init__(self, width: int, groups: int, eps: float, *, dtype, device="cpu"):
        super().__init__()
        if groups < 1 or width % groups != 0:
            raise ValueError(f"norm: {width} in {groups} groups")
        self.groups, self.eps, self.dtype = groups, float(eps), dtype
        _buffer(self, "weight", width, dtype=torch.float32, device=device)

    def rows(self, x, rows):
        return ops.group_norm_rows(x, rows, self.weight, self.groups, self.eps, self.dtype)

    def forward(self, x, y=None, alpha=1.0):
        return ops.post_norm_(x, y, alpha, self.weight, self.groups, self.eps, self.dtype)


class TokenSideInput(nn.Module):
    """What a layer adds per token: ``x += rmsnorm(proj(gelu_tanh(gate x) * e))``, e a slice of the token's row in a table
    that all layers share."""

    def __init__(self, width: int, dim: int, column: int, eps: float, *, dtype, device="cpu"):
        super().__init__()
        self.dim, self.column, self.eps = dim, column, float(eps)
        _buffer(self, "gate", dim, width, dtype=dtype, device=device)
        _buffer(self, "proj", width, dim, dtype=dtype, device=device)
        _buffer(self, "norm", width, dtype=torch.float32, device=device)

    def checkpoint(self, prefix):
        return {prefix + "gate": self.gate, prefix + "proj": self.proj, prefix + "norm": self.norm}

    def forward(self, x, h, tokens, table):
        g = ops.linear_gelu_table(h, self.gate, tokens, table, self.column)
        return ops.add_normed_(x, ops.linear(g, self.proj, torch.float32), self.norm, self.eps, h.dtype)


class ConvNorm(nn.Module):
    """RMS norm of the residual stream, then ``h + causal_conv(h)``: what a sub-layer reads."""

    def __init__(self, width: int, taps: int, eps: float, *, dtype, device="cpu"):
        super().__init__()
        self.eps, self.taps, self.dtype = float(eps), taps, dtype
        _buffer(self, "weight", width, dtype=torch.float32, device=device)
        _buffer(self, "conv", taps, width, dtype=torch.float32, device=device)   # the checkpoint's [width, taps], transposed

    def checkpoint(self, norm, conv):
        return {norm: self.weight, conv: self.conv.t()}

    def state_shape(self):
        return (self.taps - 1, self.weight.numel())

    def forward(self, x, state, step):
        return ops.rmsnorm_conv(x, self.weight, self.conv, state, step, self.eps, self.dtype)
