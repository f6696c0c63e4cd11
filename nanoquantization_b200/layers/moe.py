"""The mixture-of-experts kernels, bound through the C ABI (``include/nqb200_moe.h``).

A ``Plan`` is what routing leaves of a step: every token's experts and weights, and the (token, expert) pairs sorted by
expert.  It stays on the device; nothing of it is read by the host."""
from __future__ import annotations

import ctypes

import torch

from .. import _lib
from .mixers import DECODE_TOKENS


def _call(name: str, *args) -> None:
    _lib.check_mixers(getattr(_lib.load_moe(), name)(*args, _lib.stream_ptr()))


class Plan:
    def __init__(self, tokens: int, router: _lib.RouterDesc, device):
        pairs, experts = tokens * router.top, router.experts
        self.tokens, self.router = tokens, router
        self._ints = torch.empty(2 * pairs + 4 * experts + 2, dtype=torch.int32, device=device)
        self.expert, self.order, self.offsets, self.active, counters = self._ints.split([pairs, pairs, experts + 1, experts + 1, 2 * experts])
        self.weight = torch.empty(pairs, dtype=torch.float32, device=device)
        self.desc = _lib.MoePlan(self.expert.data_ptr(), self.weight.data_ptr(), self.offsets.data_ptr(), self.order.data_ptr(),
                                 self.active.data_ptr(), counters.data_ptr())


def route(logits: torch.Tensor, router: _lib.RouterDesc) -> Plan:
    """``logits [tokens, experts]`` float32 -> each token's experts and weights, sorted by expert."""
    _lib.require_cuda(logits)
    plan = Plan(logits.shape[0], router, logits.device)
    _call("nqb200_moe_route", logits.data_ptr(), ctypes.byref(router), ctypes.byref(plan.desc), plan.tokens)
    return plan


def _linear(x, weight, out, kind, plan):
    _call("nqb200_moe_linear", x.data_ptr(), weight.data_ptr(), out.data_ptr(), kind, plan.tokens, weight.shape[1], weight.shape[2],
          ctypes.byref(plan.router), ctypes.byref(plan.desc), _lib.mixer_dtype_code(x.dtype), _lib.mixer_dtype_code(out.dtype),
          _lib.mixer_status(x.device).data_ptr())
    return out


def experts_up(x: torch.Tensor, weight: torch.Tensor, plan: Plan) -> torch.Tensor:
    """gelu of every pair's first linear, ``weight [experts, ff, width]``; rows in the plan's order."""
    return _linear(x, weight, torch.empty(plan.tokens * plan.router.top, weight.shape[1], dtype=x.dtype, device=x.device), _lib.MOE_UP, plan)


def experts_down(u: torch.Tensor, weight: torch.Tensor, plan: Plan) -> torch.Tensor:
    """Every pair's second linear times its weight, ``weight [experts, width, ff]`` -> ``[tokens, top, width]``: float32, or
    bfloat16 in steps of more tokens than a decode step has."""
    dtype = torch.float32 if plan.tokens <= DECODE_TOKENS else u.dtype
    out = torch.empty(plan.tokens, plan.router.top, weight.shape[1], dtype=dtype, device=u.device)
    return _linear(u, weight, out, _lib.MOE_DOWN, plan)
