"""The sequence-mixing kernels, one call each, bound through the C ABI (``include/nqb200_mixers.h``).

``step`` is an engine step (``engine.batch.StepBatch``): which tokens belong to which sequence, where they stand,
which K/V blocks and which state slot the sequence owns.  The residual stream ``x`` is float32; activations are
bfloat16, or float32 when the model runs in 32 bits."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .. import _lib


def _call(name: str, *args) -> None:
    _lib.check_mixers(getattr(_lib.load_mixers(), name)(*args, _lib.stream_ptr()))


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def stream_add(x: torch.Tensor, ids: Optional[torch.Tensor], embed: Optional[torch.Tensor], step_vector: Optional[torch.Tensor],
               accumulate: bool) -> torch.Tensor:
    """In place: ``x = (x if accumulate) + embed[ids] + step_vector``."""
    _lib.require_cuda(x)
    dtype = _lib.F32 if embed is None else _lib.mixer_dtype_code(embed.dtype)
    _call("nqb200_stream_add", x.data_ptr(), _ptr(ids), _ptr(embed), _ptr(step_vector), int(accumulate), x.shape[0], x.shape[1], dtype)
    return x


def rmsnorm_rows(x: torch.Tensor, rows: Optional[torch.Tensor], weight: torch.Tensor, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """RMS norm of the given rows of the residual stream (all of them if ``rows`` is None)."""
    _lib.require_cuda(x, weight)
    out = torch.empty(x.shape[0] if rows is None else rows.numel(), x.shape[1], dtype=dtype, device=x.device)
    _call("nqb200_rmsnorm_rows", x.data_ptr(), _ptr(rows), weight.data_ptr(), out.data_ptr(), out.shape[0], out.shape[1], eps,
          _lib.mixer_dtype_code(dtype))
    return out


def group_norm_rows(x: torch.Tensor, rows: Optional[torch.Tensor], weight: torch.Tensor, groups: int, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """RMS norm in groups of the given rows of the residual stream (all of them if ``rows`` is None)."""
    _lib.require_cuda(x, weight)
    out = torch.empty(x.shape[0] if rows is None else rows.numel(), x.shape[1], dtype=dtype, device=x.device)
    _call("nqb200_group_norm_rows", x.data_ptr(), _ptr(rows), weight.data_ptr(), out.data_ptr(), out.shape[0], out.shape[1], groups, eps,
          _lib.mixer_dtype_code(dtype))
    return out


def post_norm_(x: torch.Tensor, y: Optional[torch.Tensor], alpha: float, weight: torch.Tensor, groups: int, eps: float,
               dtype: torch.dtype) -> torch.Tensor:
    """In place ``x = norm(alpha * x + y)`` (``y [tokens, terms, width]`` is summed over its terms, or None); returns the
    result rounded to ``dtype``."""
    _lib.require_cuda(x, weight)
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    _call("nqb200_post_norm", x.data_ptr(), _ptr(y), _lib.F32 if y is None else _lib.mixer_dtype_code(y.dtype), 0 if y is None else y.shape[1], alpha,
          weight.data_ptr(), h.data_ptr(), x.shape[0], x.shape[1], groups, eps, _lib.mixer_dtype_code(dtype))
    return h


def add_normed_(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """In place ``x += y / rms(y) * weight``; returns the sum rounded to ``dtype``."""
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    _call("nqb200_add_normed", x.data_ptr(), y.data_ptr(), weight.data_ptr(), h.data_ptr(), x.shape[0], x.shape[1], eps, _lib.mixer_dtype_code(dtype))
    return h


def linear_gelu_table(x: torch.Tensor, weight: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, column: int) -> torch.Tensor:
    """``gelu_tanh(x @ weight.T) * table[ids, column:column + dim]``."""
    dim = weight.shape[0]
    out = torch.empty(x.shape[0], dim, dtype=x.dtype, device=x.device)
    if decode_sized(x, weight):
        _call("nqb200_dense_decode_gelu_table", x.data_ptr(), weight.data_ptr(), ids.data_ptr(), table.data_ptr(), table.stride(0), column,
              out.data_ptr(), x.shape[0], dim, weight.shape[1])
        return out
    gate = linear(x, weight)
    _call("nqb200_gelu_table", gate.data_ptr(), ids.data_ptr(), table.data_ptr(), table.stride(0), column, out.data_ptr(), x.shape[0], dim,
          _lib.mixer_dtype_code(x.dtype))
    return out


def rmsnorm_conv(x: torch.Tensor, weight: torch.Tensor, conv: torch.Tensor, state: torch.Tensor, step, eps: float,
                 dtype: torch.dtype) -> torch.Tensor:
    """``h + causal_conv(h)`` with ``h`` the RMS norm of ``x``; ``conv [taps, width]``; ``state [slots, taps - 1, width]``
    carries the last h."""
    _lib.require_cuda(x, weight, conv)
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    _call("nqb200_rmsnorm_conv", x.data_ptr(), weight.data_ptr(), conv.data_ptr(), _ptr(state), out.data_ptr(), ctypes.byref(step.desc),
          x.shape[1], conv.shape[0], eps, _lib.mixer_dtype_code(dtype))
    return out


def rope_store(proj: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, inv_freq: torch.Tensor, step, q_off: int, k_off: int,
               v_off: int, heads: int) -> None:
    """Rotate q (in place) and k, and store k and v of every token in its cache row."""
    kv_heads, dim, vdim = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    _call("nqb200_rope_store", proj.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), _ptr(inv_freq), ctypes.byref(step.desc),
          proj.stride(0), q_off, k_off, v_off, heads, kv_heads, dim, vdim, 2 * inv_freq.numel(), _lib.mixer_dtype_code(proj.dtype))


def norm_rope(proj: torch.Tensor, k_cache: Optional[torch.Tensor], v_cache: Optional[torch.Tensor], desc: _lib.RopeDesc, step, q_off: int,
              k_off: int, v_off: int) -> None:
    """Norm (where the descriptor has weights) and rotate q in place and k; k and v of every token go to their cache row,
    or k stays in place where there is no cache."""
    _call("nqb200_norm_rope", proj.data_ptr(), _ptr(k_cache), _ptr(v_cache), ctypes.byref(desc), ctypes.byref(step.desc), proj.stride(0),
          q_off, k_off, v_off, _lib.mixer_dtype_code(proj.dtype))


def chunk_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, desc: _lib.AttentionDesc, step) -> None:
    """Attention over the paged cache; ``q`` and ``out`` are column ranges of row-major buffers."""
    _call("nqb200_chunk_attention", q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
          k_cache.shape[0] * k_cache.shape[1], ctypes.byref(desc), ctypes.byref(step.desc), _lib.mixer_status(q.device).data_ptr(), _lib.mixer_dtype_code(q.dtype))


def retention(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, decay: Optional[torch.Tensor], state: torch.Tensor, step,
              log_decay: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``o [tokens, heads, vdim]`` float32; ``state [slots, heads, dim, vdim]`` is carried.  ``decay [heads]``, or
    ``log_decay [tokens, heads * dim]`` where every key channel of every token has its own."""
    _, heads, dim, vdim = state.shape
    o = torch.empty(proj.shape[0], heads, vdim, dtype=torch.float32, device=proj.device)
    _call("nqb200_retention", proj.data_ptr(), proj.stride(0), q_off, k_off, v_off, _ptr(decay), _ptr(log_decay), state.data_ptr(), o.data_ptr(),
          heads, dim, vdim, ctypes.byref(step.desc), _lib.mixer_dtype_code(proj.dtype))
    return o


def gla_log_decay(low: torch.Tensor, a2: torch.Tensor, bias: torch.Tensor, tau: float) -> torch.Tensor:
    """``log(sigmoid(low @ a2.T + bias)) / tau`` in float32; ``low`` is a column range."""
    out = torch.empty(low.shape[0], a2.shape[0], dtype=torch.float32, device=low.device)
    _call("nqb200_gla_log_decay", low.data_ptr(), low.stride(0), a2.data_ptr(), bias.data_ptr(), out.data_ptr(), low.shape[0], a2.shape[0],
          a2.shape[1], tau, _lib.mixer_dtype_code(low.dtype))
    return out


def head_norm_gate(o: torch.Tensor, gate: torch.Tensor, out: torch.Tensor, eps: float, out_scale: float, weight: Optional[torch.Tensor] = None) -> None:
    """``out = out_scale * o / rms(o) * weight * silu(gate)`` per head; ``gate`` and ``out`` are column ranges."""
    T, heads, vdim = o.shape
    _call("nqb200_head_norm_gate", o.data_ptr(), gate.data_ptr(), gate.stride(0), _ptr(weight), out.data_ptr(), out.stride(0), T, heads, vdim, eps,
          out_scale, _lib.mixer_dtype_code(out.dtype))


RETENTION_PREFILL_TOKENS = 17   # shorter portions take the token-by-token kernel


def retention_gated(proj: torch.Tensor, off: int, desc: _lib.RetentionDesc, decay: torch.Tensor, state: torch.Tensor, act: torch.Tensor,
                    act_col: int, step) -> None:
    """Retention with norm and gate: ``proj`` holds q | k | v | gate from column ``off``, the result goes to ``act``
    from column ``act_col``.  Prompts in bfloat16 run chunkwise on the tensor cores, the rest token by token."""
    lib = _lib.load_mixers()
    _, heads, dim, vdim = state.shape
    if (proj.dtype == torch.bfloat16 and step.max_len >= RETENTION_PREFILL_TOKENS
            and lib.nqb200_retention_prefill_supported(ctypes.byref(desc), proj.stride(0), off, act.stride(0), act_col)):
        chunks = lib.nqb200_retention_chunks(step.num_tokens, step.batch)
        scratch = torch.empty(2, chunks, heads, dim, vdim, dtype=torch.float32, device=proj.device)
        _call("nqb200_retention_prefill", proj.data_ptr(), proj.stride(0), off, act.data_ptr(), act.stride(0), act_col, ctypes.byref(desc),
              state.data_ptr(), scratch.data_ptr(), ctypes.byref(step.desc))
        return
    k_off, v_off = off + heads * dim, off + 2 * heads * dim
    g_off = v_off + heads * vdim
    o = retention(proj, off, k_off, v_off, decay, state, step)
    head_norm_gate(o, proj[:, g_off:g_off + heads * vdim], act[:, act_col:act_col + heads * vdim], desc.eps, desc.out_scale)


def gla_gated(proj: torch.Tensor, off: int, m, state: torch.Tensor, act: torch.Tensor, act_col: int, step) -> None:
    """Gated linear attention with norm and gate of mixer ``m``: ``proj`` holds q | k | v | gate | low-rank decay input from
    column ``off``, the result goes to ``act`` from column ``act_col``.  Prompts in bfloat16 run chunkwise on the tensor cores,
    the rest token by token."""
    _, heads, dim, vdim = state.shape
    k_off, v_off = off + heads * dim, off + 2 * heads * dim
    g_off = v_off + heads * vdim
    a_off = g_off + heads * vdim
    lib, desc = _lib.load_mixers(), m.desc()
    if (proj.dtype == torch.bfloat16 and step.max_len >= RETENTION_PREFILL_TOKENS
            and lib.nqb200_gla_prefill_supported(ctypes.byref(desc), proj.stride(0), off, act.stride(0), act_col)):
        scratch = torch.empty(lib.nqb200_gla_scratch(ctypes.byref(desc), step.num_tokens, step.batch), dtype=torch.float32, device=proj.device)
        _call("nqb200_gla_prefill", proj.data_ptr(), proj.stride(0), off, act.data_ptr(), act.stride(0), act_col, ctypes.byref(desc),
              state.data_ptr(), scratch.data_ptr(), ctypes.byref(step.desc))
        return
    log_decay = gla_log_decay(proj[:, a_off:a_off + m.rank], m.a2, m.a2_bias, m.tau)
    o = retention(proj, off, k_off, v_off, None, state, step, log_decay)
    head_norm_gate(o, proj[:, g_off:a_off], act[:, act_col:act_col + heads * vdim], m.eps, m.out_scale, m.norm)


def mingru(proj: torch.Tensor, width: int, z_bias: torch.Tensor, x_bias: torch.Tensor, state: torch.Tensor, step) -> torch.Tensor:
    """``proj [tokens, z | x | g]`` -> gated states ``[tokens, width]``; ``state [slots, width]`` is carried."""
    out = torch.empty(proj.shape[0], width, dtype=proj.dtype, device=proj.device)
    scratch = None
    if step.max_len > 128:
        scratch = torch.empty(_lib.load_mixers().nqb200_mingru_scratch(step.num_tokens, step.batch, width), dtype=torch.float32, device=proj.device)
    _call("nqb200_mingru", proj.data_ptr(), proj.stride(0), 0, width, 2 * width, z_bias.data_ptr(), x_bias.data_ptr(), state.data_ptr(),
          out.data_ptr(), width, _ptr(scratch), ctypes.byref(step.desc), _lib.mixer_dtype_code(proj.dtype))
    return out


def clamped_glu(gate_up: torch.Tensor, limit: float) -> torch.Tensor:
    T, two_ff = gate_up.shape
    out = torch.empty(T, two_ff // 2, dtype=gate_up.dtype, device=gate_up.device)
    _call("nqb200_clamped_glu", gate_up.data_ptr(), out.data_ptr(), T, two_ff // 2, limit, _lib.mixer_dtype_code(gate_up.dtype))
    return out


DECODE_TOKENS = 16   # up to here the linears run as kernels that stream the weights once


def decode_sized(x: torch.Tensor, weight: torch.Tensor) -> bool:
    return x.dtype == torch.bfloat16 and 0 < x.shape[0] <= DECODE_TOKENS and weight.shape[1] % 8 == 0


def _dense(x, weight, out, mode, beta=0.0):
    _call("nqb200_dense_decode", x.data_ptr(), weight.data_ptr(), out.data_ptr(), x.shape[0], weight.shape[0], weight.shape[1], mode, beta)
    return out


def linear(x: torch.Tensor, weight: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``x @ weight.T`` with 32-bit accumulation: the streaming kernel for decode sizes, a library product otherwise."""
    dtype = out_dtype or x.dtype
    if decode_sized(x, weight):
        out = torch.empty(x.shape[0], weight.shape[0], dtype=dtype, device=x.device)
        return _dense(x, weight, out, _lib.DENSE_F32 if dtype == torch.float32 else _lib.DENSE_BF16)
    if x.dtype == dtype:
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out_dtype=dtype)


def linear_residual_(stream: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, beta: float = 1.0) -> torch.Tensor:
    """``stream = beta * stream + y @ weight.T``: the product is added to the float32 stream before any rounding."""
    if decode_sized(y, weight):
        return _dense(y, weight, stream, _lib.DENSE_RESIDUAL, beta)
    if y.dtype == torch.float32:
        return stream.addmm_(y, weight.t(), beta=beta)
    return torch.addmm(stream, y, weight.t(), out_dtype=torch.float32, beta=beta, out=stream)


def dense_glu(x: torch.Tensor, weight: torch.Tensor, limit: float) -> torch.Tensor:
    """Decode sizes: the merged gate | up product with the clamped GLU inside."""
    out = torch.empty(x.shape[0], weight.shape[0] // 2, dtype=x.dtype, device=x.device)
    _call("nqb200_dense_decode_glu", x.data_ptr(), weight.data_ptr(), out.data_ptr(), x.shape[0], out.shape[1], weight.shape[1], limit)
    return out


def dense_mingru(x: torch.Tensor, weight: torch.Tensor, z_bias: torch.Tensor, x_bias: torch.Tensor, state: torch.Tensor, step) -> torch.Tensor:
    """Decode sizes, one token per sequence: the merged z | x | g product with the minGRU update inside."""
    width = weight.shape[0] // 3
    out = torch.empty(x.shape[0], width, dtype=x.dtype, device=x.device)
    _call("nqb200_dense_decode_mingru", x.data_ptr(), weight.data_ptr(), z_bias.data_ptr(), x_bias.data_ptr(), state.data_ptr(), out.data_ptr(),
          width, weight.shape[1], ctypes.byref(step.desc))
    return out


def mixer_decode_supported(att: Optional[_lib.AttentionDesc], ret: Optional[_lib.RetentionDesc]) -> bool:
    lib = _lib.load_mixers()
    return bool(lib.nqb200_mixer_decode_supported(None if att is None else ctypes.byref(att), None if ret is None else ctypes.byref(ret)))


def mixer_decode(proj: torch.Tensor, act: torch.Tensor, att, ret, step) -> None:
    """One token per sequence, attention and retention (or gated linear attention) in one launch.  ``att = (desc, rope desc,
    first projection column, column of the values, first output column, k_cache, v_cache)``, ``ret = (desc, first
    projection column, first output column, state)``; either may be None."""
    a = (None, None, 0, 0, 0, None, None) if att is None else (
        ctypes.byref(att[0]), ctypes.byref(att[1]), att[2], att[3], att[4], att[5].data_ptr(), att[6].data_ptr())
    r = (None, 0, 0, None) if ret is None else (ctypes.byref(ret[0]), ret[1], ret[2], ret[3].data_ptr())
    _call("nqb200_mixer_decode", proj.data_ptr(), proj.stride(0), act.data_ptr(), act.stride(0), *a, *r, ctypes.byref(step.desc))
