"""ctypes binding of libnqb200.so (the C ABI declared in include/nqb200.h).

There is no fallback: if the shared library is missing, or a call returns a
nonzero status, a RuntimeError is raised.
"""
from __future__ import annotations

import ctypes
import os
import threading

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "lib", "libnqb200.so")
MIXERS_PATH = os.path.join(_HERE, "lib", "libnqb200_mixers.so")
MOE_PATH = os.path.join(_HERE, "lib", "libnqb200_moe.so")

F16, BF16, F32 = 0, 1, 2
_vp, _i64, _int, _sz = ctypes.c_void_p, ctypes.c_int64, ctypes.c_int, ctypes.c_size_t

class DecodeFusion(ctypes.Structure):
    """nqb200_decode_fusion of include/nqb200.h."""
    _fields_ = [("norm_ssq", ctypes.c_void_p), ("norm_tiles", ctypes.c_int64), ("norm_weight", ctypes.c_void_p),
                ("norm_eps", ctypes.c_float), ("silu_mul", ctypes.c_int), ("residual_in", ctypes.c_void_p),
                ("ssq_out", ctypes.c_void_p)]


FUSE_RMSNORM, FUSE_RESIDUAL, FUSE_SILU_MUL, FUSE_ALLREDUCE = 1, 2, 4, 8

# name -> (restype, argtypes); mirrors include/nqb200.h one to one
SIGNATURES = {
    "nqb200_version": (_int, []),
    "nqb200_status_string": (ctypes.c_char_p, [_int]),
    "nqb200_device_supported": (_int, [_int]),
    "nqb200_unpack_int4": (_int, [_vp, _vp, _i64, _i64, _vp]),
    "nqb200_dequant": (_int, [_vp, _vp, _vp, _vp, _i64, _i64, _i64, _int, _vp]),
    "nqb200_gemm_workspace_bytes": (_sz, [_i64, _i64, _i64, _i64, _int]),
    "nqb200_gemm": (_int, [_vp, _vp, _vp, _vp, _vp, _int, _vp, _i64, _i64, _i64, _i64, _int, _vp, _sz, _vp]),
    "nqb200_decode_tile_columns": (_int, []),
    "nqb200_gemm_gate_up_silu_supported": (_int, [_i64, _i64, _i64, _i64, _int]),
    "nqb200_gemm_gate_up_silu": (_int, [_vp, _vp, _vp, _vp, _vp, _int, _vp, _i64, _i64, _i64, _i64, _int, _vp, _sz, _vp]),
    "nqb200_gemm_decode_fused_supported": (_int, [_i64, _i64, _i64, _i64, _int, _int, _int, _sz]),
    "nqb200_gemm_decode_fused": (_int, [_vp, _vp, _vp, _vp, _vp, _int, _vp, _i64, _i64, _i64, _i64, _int, _vp, _sz,
                                 ctypes.POINTER(DecodeFusion), ctypes.POINTER(_vp), _int, _int, _sz, _sz, _vp]),
    "nqb200_gemm_decode_noalloc": (_int, [_vp, _vp, _vp, _vp, _vp, _int, _vp, _i64, _i64, _i64, _i64, _int, _vp]),
    "nqb200_quantize_pack": (_int, [_vp, _int, _vp, _vp, _vp, _i64, _i64, _i64, _int, _vp]),
    "nqb200_add_rmsnorm": (_int, [_vp, _vp, _vp, _vp, _vp, _i64, _i64, ctypes.c_float, _int, _vp]),
    "nqb200_qknorm_rope": (_int, [_vp, _vp, _vp, _vp, _vp, _i64, _i64, _i64, _i64, _i64, ctypes.c_float, _int, _vp]),
    "nqb200_qknorm_rope_kv": (_int, [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _i64, _i64, _i64, ctypes.c_float, _int, _vp]),
    "nqb200_silu_mul": (_int, [_vp, _vp, _i64, _i64, _int, _vp]),
    "nqb200_comm_alloc": (_int, [ctypes.POINTER(_vp), _sz]),
    "nqb200_comm_free": (_int, [_vp]),
    "nqb200_comm_export": (_int, [_vp, _vp]),
    "nqb200_comm_import": (_int, [_vp, ctypes.POINTER(_vp)]),
    "nqb200_comm_unimport": (_int, [_vp]),
    "nqb200_comm_data_offset": (_sz, []),
    "nqb200_comm_set_wait_limit": (_int, [_vp, ctypes.c_uint64]),
    "nqb200_comm_status": (_int, [_vp, _vp]),
    "nqb200_gemm_allreduce_supported": (_int, [_i64, _i64, _i64, _i64, _int, _int, _sz]),
    "nqb200_gemm_allreduce": (_int, [_vp, _vp, _vp, _vp, _vp, _int, _vp, _i64, _i64, _i64, _i64, _int, _vp, _sz, ctypes.POINTER(_vp), _int, _int, _sz, _sz, _vp]),
    "nqb200_peer_allreduce": (_int, [ctypes.POINTER(_vp), _int, _int, _sz, _vp, _vp, _int, _i64, _i64, _int, _vp]),
    "nqb200_peer_allreduce_large": (_int, [ctypes.POINTER(_vp), _int, _int, _sz, _sz, _vp, _vp, _int, _i64, _i64, _int, _vp]),
    "nqb200_workspace_status": (_int, [_vp, _sz, _vp]),
    "nqb200_gemm_kernel_name": (ctypes.c_char_p, [_i64, _i64, _i64, _i64, _int]),
    "nqb200_gemm_launch_count": (_int, [_i64, _i64, _i64, _i64, _int]),
}


class StepDesc(ctypes.Structure):
    """nqb200_batch of include/nqb200_mixers.h."""
    _fields_ = [("cu", _vp), ("pos0", _vp), ("slot", _vp), ("table", _vp), ("batch", ctypes.c_int32), ("tokens", ctypes.c_int32),
                ("max_len", ctypes.c_int32), ("table_width", ctypes.c_int32), ("block_size", ctypes.c_int32)]


class AttentionDesc(ctypes.Structure):
    """nqb200_attention of include/nqb200_mixers.h."""
    _fields_ = [("heads", ctypes.c_int32), ("kv_heads", ctypes.c_int32), ("dim", ctypes.c_int32), ("vdim", ctypes.c_int32),
                ("chunk", ctypes.c_int32), ("scale", ctypes.c_float), ("softcap", ctypes.c_float), ("sink", _vp),
                ("out_scale", ctypes.c_float), ("temp", _vp), ("bias", _vp), ("sigmoid", ctypes.c_int32)]


class RopeDesc(ctypes.Structure):
    """nqb200_rope of include/nqb200_mixers.h."""
    _fields_ = [("heads", ctypes.c_int32), ("kv_heads", ctypes.c_int32), ("dim", ctypes.c_int32), ("vdim", ctypes.c_int32),
                ("rot", ctypes.c_int32), ("interleaved", ctypes.c_int32), ("inv_freq", _vp), ("q_norm", _vp), ("k_norm", _vp),
                ("eps", ctypes.c_float)]


class RetentionDesc(ctypes.Structure):
    """nqb200_retention_desc of include/nqb200_mixers.h."""
    _fields_ = [("heads", ctypes.c_int32), ("dim", ctypes.c_int32), ("vdim", ctypes.c_int32), ("eps", ctypes.c_float),
                ("out_scale", ctypes.c_float), ("decay", _vp), ("norm", _vp), ("inv_freq", _vp), ("rot", ctypes.c_int32),
                ("rank", ctypes.c_int32), ("tau", ctypes.c_float), ("a2", _vp), ("a2_bias", _vp)]


class RouterDesc(ctypes.Structure):
    """nqb200_router of include/nqb200_moe.h."""
    _fields_ = [("experts", ctypes.c_int32), ("top", ctypes.c_int32), ("groups", ctypes.c_int32), ("keep", ctypes.c_int32),
                ("scale", ctypes.c_float), ("correction", _vp)]


class MoePlan(ctypes.Structure):
    """nqb200_moe_plan of include/nqb200_moe.h."""
    _fields_ = [("expert", _vp), ("weight", _vp), ("offsets", _vp), ("order", _vp), ("active", _vp), ("counters", _vp)]


MOE_UP, MOE_DOWN = 0, 1
DENSE_BF16, DENSE_F32, DENSE_RESIDUAL = 0, 1, 2
_ret = ctypes.POINTER(RetentionDesc)
_step, _att, _f32 = ctypes.POINTER(StepDesc), ctypes.POINTER(AttentionDesc), ctypes.c_float
_rope, _router, _plan = ctypes.POINTER(RopeDesc), ctypes.POINTER(RouterDesc), ctypes.POINTER(MoePlan)
# mirrors include/nqb200_mixers.h one to one
MIXER_SIGNATURES = {
    "nqb200_stream_add": (_int, [_vp, _vp, _vp, _vp, _int, _i64, _i64, _int, _vp]),
    "nqb200_rmsnorm_rows": (_int, [_vp, _vp, _vp, _vp, _i64, _i64, _f32, _int, _vp]),
    "nqb200_group_norm_rows": (_int, [_vp, _vp, _vp, _vp, _i64, _i64, _i64, _f32, _int, _vp]),
    "nqb200_post_norm": (_int, [_vp, _vp, _int, _i64, _f32, _vp, _vp, _i64, _i64, _i64, _f32, _int, _vp]),
    "nqb200_gelu_table": (_int, [_vp, _vp, _vp, _i64, _i64, _vp, _i64, _i64, _int, _vp]),
    "nqb200_add_normed": (_int, [_vp, _vp, _vp, _vp, _i64, _i64, _f32, _int, _vp]),
    "nqb200_rmsnorm_conv": (_int, [_vp, _vp, _vp, _vp, _vp, _step, _i64, _i64, _f32, _int, _vp]),
    "nqb200_rope_store": (_int, [_vp, _vp, _vp, _vp, _step] + [_i64] * 9 + [_int, _vp]),
    "nqb200_norm_rope": (_int, [_vp, _vp, _vp, _rope, _step, _i64, _i64, _i64, _i64, _int, _vp]),
    "nqb200_chunk_attention": (_int, [_vp, _i64, _vp, _vp, _vp, _i64, _i64, _att, _step, _vp, _int, _vp]),
    "nqb200_retention": (_int, [_vp, _i64, _i64, _i64, _i64, _vp, _vp, _vp, _vp, _i64, _i64, _i64, _step, _int, _vp]),
    "nqb200_gla_log_decay": (_int, [_vp, _i64, _vp, _vp, _vp, _i64, _i64, _i64, _f32, _int, _vp]),
    "nqb200_head_norm_gate": (_int, [_vp, _vp, _i64, _vp, _vp, _i64, _i64, _i64, _i64, _f32, _f32, _int, _vp]),
    "nqb200_mingru": (_int, [_vp, _i64, _i64, _i64, _i64, _vp, _vp, _vp, _vp, _i64, _vp, _step, _int, _vp]),
    "nqb200_mingru_scratch": (_i64, [_i64, _i64, _i64]),
    "nqb200_clamped_glu": (_int, [_vp, _vp, _i64, _i64, _f32, _int, _vp]),
    "nqb200_retention_prefill": (_int, [_vp, _i64, _i64, _vp, _i64, _i64, _ret, _vp, _vp, _step, _vp]),
    "nqb200_retention_prefill_supported": (_int, [_ret, _i64, _i64, _i64, _i64]),
    "nqb200_retention_chunks": (_i64, [_i64, _i64]),
    "nqb200_gla_prefill": (_int, [_vp, _i64, _i64, _vp, _i64, _i64, _ret, _vp, _vp, _step, _vp]),
    "nqb200_gla_prefill_supported": (_int, [_ret, _i64, _i64, _i64, _i64]),
    "nqb200_gla_scratch": (_i64, [_ret, _i64, _i64]),
    "nqb200_dense_decode": (_int, [_vp, _vp, _vp, _i64, _i64, _i64, _int, _f32, _vp]),
    "nqb200_dense_decode_gelu_table": (_int, [_vp, _vp, _vp, _vp, _i64, _i64, _vp, _i64, _i64, _i64, _vp]),
    "nqb200_dense_decode_glu": (_int, [_vp, _vp, _vp, _i64, _i64, _i64, _f32, _vp]),
    "nqb200_dense_decode_mingru": (_int, [_vp] * 6 + [_i64, _i64, _step, _vp]),
    "nqb200_mixer_decode_supported": (_int, [_att, _ret]),
    "nqb200_mixer_decode": (_int, [_vp, _i64, _vp, _i64, _att, _rope, _i64, _i64, _i64, _vp, _vp, _ret, _i64, _i64, _vp, _step, _vp]),
}

# mirrors include/nqb200_moe.h one to one
MOE_SIGNATURES = {
    "nqb200_moe_route": (_int, [_vp, _router, _plan, _i64, _vp]),
    "nqb200_moe_linear": (_int, [_vp, _vp, _vp, _int, _i64, _i64, _i64, _router, _plan, _int, _int, _vp, _vp]),
    "nqb200_moe_linear_kernel": (ctypes.c_char_p, [_i64, _i64, _i64, _i64, _int]),
}

_lib = None
_more: dict[str, ctypes.CDLL] = {}
_lock = threading.Lock()


def load() -> ctypes.CDLL:
    """Load the library once; raise if it has not been built."""
    global _lib
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is None:
            if not os.path.exists(LIB_PATH):
                raise RuntimeError(
                    f"{LIB_PATH} is missing: build it with "
                    "`python -m nanoquantization_b200.csrc.build` (needs nvcc). "
                    "There is no CPU or PyTorch fallback for the W4A16 kernels.")
            lib = ctypes.CDLL(LIB_PATH)
            for name, (res, args) in SIGNATURES.items():
                fn = getattr(lib, name)
                fn.restype = res
                fn.argtypes = args
            _lib = lib
    return _lib


def _load_once(path: str, signatures: dict) -> ctypes.CDLL:
    lib = _more.get(path)
    if lib is None:
        with _lock:
            if path not in _more:
                if not os.path.exists(path):
                    raise RuntimeError(f"{path} is missing: build it with `python -m nanoquantization_b200.csrc.build` "
                                       "(needs nvcc). There is no CPU or PyTorch fallback for these kernels.")
                lib = ctypes.CDLL(path)
                for name, (res, args) in signatures.items():
                    fn = getattr(lib, name)
                    fn.restype, fn.argtypes = res, args
                _more[path] = lib
            lib = _more[path]
    return lib


def load_mixers() -> ctypes.CDLL:
    """Load the library of sequence-mixing kernels once; raise if it has not been built."""
    return _load_once(MIXERS_PATH, MIXER_SIGNATURES)


def load_moe() -> ctypes.CDLL:
    """Load the library of mixture-of-experts kernels once; raise if it has not been built."""
    return _load_once(MOE_PATH, MOE_SIGNATURES)


_STATUS = ("ok", "bad shape", "bad dtype", "misaligned pointer", "null pointer", "workspace missing or too small",
           "unsupported device", "CUDA launch failed", "a bounded device-side wait timed out", "size exceeds the supported maximum")


def check_mixers(status: int) -> None:
    if status != 0:
        raise RuntimeError(f"nqb200_mixers: {_STATUS[status] if status < len(_STATUS) else 'unknown status'} (status {status})")


_mixer_status: dict[int, torch.Tensor] = {}


def mixer_status(dev: torch.device) -> torch.Tensor:
    """The device's status word for bounded waits of the mixer kernels (0: none gave up)."""
    idx = dev.index if dev.index is not None else torch.cuda.current_device()
    if idx not in _mixer_status:
        _mixer_status[idx] = torch.zeros(1, dtype=torch.int32, device=dev)
    return _mixer_status[idx]


def check_mixer_status() -> None:
    """Synchronise and raise if a bounded wait of a mixer kernel gave up; the word is cleared."""
    for word in _mixer_status.values():
        status = int(word.item())
        if status != 0:
            word.zero_()
            check_mixers(status)


def mixer_dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.bfloat16:
        return BF16
    if dtype == torch.float32:
        return F32
    raise TypeError(f"the sequence-mixing kernels take bfloat16 or float32, got {dtype}")


def check(status: int) -> None:
    if status != 0:
        raise RuntimeError(f"nqb200: {load().nqb200_status_string(status).decode()} (status {status})")


def dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.float16:
        return F16
    if dtype == torch.bfloat16:
        return BF16
    raise TypeError(f"W4A16 kernels take float16 or bfloat16, got {dtype}")


def require_cuda(*tensors: torch.Tensor) -> torch.device:
    dev = tensors[0].device
    for t in tensors:
        if t.device.type != "cuda":
            raise RuntimeError("nanoquantization_b200 runs on CUDA tensors only (no CPU fallback); "
                               f"got a tensor on {t.device}")
        if t.device != dev:
            raise RuntimeError("all tensors must be on the same device")
    return dev


_supported: dict[int, bool] = {}


def require_b200(dev: torch.device) -> None:
    idx = dev.index if dev.index is not None else torch.cuda.current_device()
    ok = _supported.get(idx)
    if ok is None:
        ok = load().nqb200_device_supported(idx) == 1
        _supported[idx] = ok
    if not ok:
        check(6)


def stream_ptr() -> int:
    return torch.cuda.current_stream().cuda_stream


_workspaces: dict[tuple[int, int], torch.Tensor] = {}


def workspace(dev: torch.device, nbytes: int) -> torch.Tensor | None:
    """Zero-filled scratch, one per (device, stream), grown on demand.  The
    kernels leave it zero-filled again, so it is only cleared when created."""
    if nbytes == 0:
        return None
    key = (dev.index if dev.index is not None else torch.cuda.current_device(), stream_ptr())
    ws = _workspaces.get(key)
    if ws is None or ws.numel() < nbytes:
        ws = torch.zeros(max(nbytes, 1 << 20), dtype=torch.uint8, device=dev)
        _workspaces[key] = ws
    return ws


def check_workspaces() -> None:
    """Synchronise and raise if any kernel recorded a give-up (a bounded wait that ran out)."""
    if not _workspaces:
        return
    lib = load()
    for (_dev, stream), ws in list(_workspaces.items()):
        check(lib.nqb200_workspace_status(ws.data_ptr(), ws.numel(), stream))
