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


def rmsnorm_conv(x: torch.Tensor, weight: torch.Tensor, conv: torch.Tensor, state: torch.Tensor, step, eps: float,
                 dtype: torch.dtype) -> torch.Tensor:
    """``h + causal_conv(h)`` with ``h`` the RMS norm of ``x``; ``state [slots, taps - 1, width]`` carries the last h."""
    _lib.require_cuda(x, weight, conv)
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    _call("nqb200_rmsnorm_conv", x.data_ptr(), weight.data_ptr(), conv.data_ptr(), _ptr(state), out.data_ptr(), ctypes.byref(step.desc),
          x.shape[1], conv.shape[1], eps, _lib.mixer_dtype_code(dtype))
    return out


def rope_store(proj: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, inv_freq: torch.Tensor, step, q_off: int, k_off: int,
               v_off: int, heads: int) -> None:
    """Rotate q (in place) and k, and store k and v of every token in its cache row."""
    kv_heads, dim, vdim = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    _call("nqb200_rope_store", proj.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), _ptr(inv_freq), ctypes.byref(step.desc),
          proj.stride(0), q_off, k_off, v_off, heads, kv_heads, dim, vdim, 2 * inv_freq.numel(), _lib.mixer_dtype_code(proj.dtype))


def chunk_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, desc: _lib.AttentionDesc, step) -> None:
    """Attention over the paged cache; ``q`` and ``out`` are column ranges of row-major buffers."""
    _call("nqb200_chunk_attention", q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
          ctypes.byref(desc), ctypes.byref(step.desc), _lib.mixer_dtype_code(q.dtype))


def retention(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, decay: torch.Tensor, state: torch.Tensor, step) -> torch.Tensor:
    """``o [tokens, heads, vdim]`` float32; ``state [slots, heads, dim, vdim]`` is carried."""
    _, heads, dim, vdim = state.shape
    o = torch.empty(proj.shape[0], heads, vdim, dtype=torch.float32, device=proj.device)
    _call("nqb200_retention", proj.data_ptr(), proj.stride(0), q_off, k_off, v_off, decay.data_ptr(), state.data_ptr(), o.data_ptr(),
          heads, dim, vdim, ctypes.byref(step.desc), _lib.mixer_dtype_code(proj.dtype))
    return o


def head_norm_gate(o: torch.Tensor, gate: torch.Tensor, out: torch.Tensor, eps: float, out_scale: float) -> None:
    """``out = out_scale * o / rms(o) * silu(gate)`` per head; ``gate`` and ``out`` are column ranges."""
    T, heads, vdim = o.shape
    _call("nqb200_head_norm_gate", o.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(), out.stride(0), T, heads, vdim, eps,
          out_scale, _lib.mixer_dtype_code(out.dtype))


def mingru(proj: torch.Tensor, width: int, z_bias: torch.Tensor, x_bias: torch.Tensor, state: torch.Tensor, step) -> torch.Tensor:
    """``proj [tokens, z | x | g]`` -> gated states ``[tokens, width]``; ``state [slots, width]`` is carried."""
    out = torch.empty(proj.shape[0], width, dtype=proj.dtype, device=proj.device)
    _call("nqb200_mingru", proj.data_ptr(), proj.stride(0), 0, width, 2 * width, z_bias.data_ptr(), x_bias.data_ptr(), state.data_ptr(),
          out.data_ptr(), width, ctypes.byref(step.desc), _lib.mixer_dtype_code(proj.dtype))
    return out


def clamped_glu(gate_up: torch.Tensor, limit: float) -> torch.Tensor:
    T, two_ff = gate_up.shape
    out = torch.empty(T, two_ff // 2, dtype=gate_up.dtype, device=gate_up.device)
    _call("nqb200_clamped_glu", gate_up.data_ptr(), out.data_ptr(), T, two_ff // 2, limit, _lib.mixer_dtype_code(gate_up.dtype))
    return out


def linear(x: torch.Tensor, weight: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``x @ weight.T`` with 32-bit accumulation."""
    if x.dtype == torch.float32 or out_dtype in (None, x.dtype):
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out_dtype=out_dtype)


def linear_residual_(stream: torch.Tensor, y: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``stream += y @ weight.T``: the product is added to the float32 stream before any rounding."""
    if y.dtype == torch.float32:
        return stream.addmm_(y, weight.t())
    return torch.addmm(stream, y, weight.t(), out_dtype=torch.float32, out=stream)
