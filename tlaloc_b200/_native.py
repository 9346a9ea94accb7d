"""ctypes binding of libtlaloc_kernels.so (the C ABI in include/tlaloc_b200.h).

There is no fallback: if the library is missing and cannot be built, importing the ops raises.
"""
from __future__ import annotations

import ctypes
import os
import re

from . import build as _build

F32, BF16, S8, S32, F8E4M3FN = 11, 16, 2, 4, 20
OK, INVALID_ARGUMENT, UNSUPPORTED, INTERNAL = 0, -1, -2, -3
GEMM_EXACT, GEMM_X_F32_EXACT, GEMM_WEIGHTS_CONST, GEMM_I8_MMA, GEMM_X_PLANES = 1, 2, 4, 8, 16

ACT_NONE, ACT_RELU2, ACT_SILU_MUL, ACT_GELU_TANH_MUL = 0, 1, 2, 3

_lib = None
_subset: str | None = None

_vp, _i32, _f32, _sz = ctypes.c_void_p, ctypes.c_int32, ctypes.c_float, ctypes.c_size_t

_i64 = ctypes.c_int64


class DenseProblem(ctypes.Structure):
    """tlaloc_b200_dense_problem"""
    _fields_ = [("x", _vp), ("w", _vp), ("bias", _vp), ("residual", _vp), ("y", _vp),
                ("ld_x", _i64), ("ld_res", _i64), ("ld_y", _i64), ("batch_x", _i64), ("batch_w", _i64), ("batch_y", _i64),
                ("k", _i32), ("n", _i32), ("batch", _i32), ("act", _i32), ("y_dtype", _i32), ("rows", _i32), ("row_offsets", _vp)]


class RotatePart(ctypes.Structure):
    """tlaloc_b200_rotate_part"""
    _fields_ = [("out", _vp), ("out_ld", _i64), ("out_head_ld", _i64), ("first", _i32), ("heads", _i32), ("dim", _i32), ("padded", _i32),
                ("rotate", _i32), ("by_slot", _i32), ("scale", _f32)]


_SIGNATURES = {
    "tlaloc_b200_abi_version": (ctypes.c_int, []),
    "tlaloc_b200_last_error": (ctypes.c_char_p, []),
    "tlaloc_b200_init": (ctypes.c_int, []),
    "tlaloc_b200_launch_count": (ctypes.c_longlong, []),
    "tlaloc_b200_device_status": (ctypes.c_int, []),
    "tlaloc_b200_set_order_faithful": (ctypes.c_int, [ctypes.c_int]),
    "tlaloc_b200_paged_attention_splits": (ctypes.c_int, [_i32] * 5),
    "tlaloc_b200_paged_attention_scratch_bytes": (_sz, [_i32] * 4),
    "tlaloc_b200_paged_attention": (ctypes.c_int, [_vp, _i32, _vp, _vp, _i32, _vp, _vp, _vp, _i32, _vp, _i32, _vp, _vp,
                                                   _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _f32, _i32,
                                                   _vp]),
    "tlaloc_b200_paged_attention_static_scratch_bytes": (_sz, []),
    "tlaloc_b200_paged_attention_static": (ctypes.c_int, [_vp, _i32, _vp, _vp, _i32, _vp, _vp, _vp, _i32, _vp, _i32, _vp,
                                                          _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _f32, _i32,
                                                          _vp]),
    "tlaloc_b200_kv_cache_write": (ctypes.c_int, [_vp, _i32, _vp, _i32, _vp, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_int8_gemm_scratch_bytes": (_sz, [_i32] * 3),
    "tlaloc_b200_int8_gemm": (ctypes.c_int, [_vp, _i32, _vp, _vp, _vp, _vp, _i32, _vp, _sz, _i32, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_int8_gemm_swiglu": (ctypes.c_int, [_vp, _i32, _vp, _vp, _vp, _i32, _vp, _sz, _i32, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_dense_gemm_exact": (ctypes.c_int, [_vp, _i32, _vp, _i32, _vp, _i32, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_embedding": (ctypes.c_int, [_vp, _i32, _vp, _vp, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_rmsnorm": (ctypes.c_int, [_vp, _vp, _vp, _i32, _i32, _i32, _f32, _vp]),
    "tlaloc_b200_rmsnorm_planes": (ctypes.c_int, [_vp, _vp, _vp, _vp, _sz, _i32, _i32, _f32, _vp]),
    "tlaloc_b200_rope_kv_write": (ctypes.c_int, [_vp] * 8 + [_i32, _vp, _vp, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_swiglu": (ctypes.c_int, [_vp, _vp, _i32, _vp, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_argmax": (ctypes.c_int, [_vp, _vp, _i32, _i32, _vp]),
    "tlaloc_b200_dense_gemm": (ctypes.c_int, [ctypes.POINTER(DenseProblem), _i32, _i32, _i32, _i32, _vp]),
    "tlaloc_b200_rmsnorm_pair": (ctypes.c_int, [_vp, _vp, _vp, _vp, _vp, _i32, _i32, _i32, _f32, _vp]),
    "tlaloc_b200_latent_kv_write": (ctypes.c_int, [_vp, _i64, _vp, _vp, _f32, _vp, _vp, _vp, _vp, _vp, _vp, _i32, _i64] + [_i32] * 7 + [_vp]),
    "tlaloc_b200_rope_interleaved": (ctypes.c_int, [_vp, _i64, _i64, _vp, _i64, _i64, _i32, _vp, _vp, _vp] + [_i32] * 5 + [_vp]),
    "tlaloc_b200_latent_attention_scratch_bytes": (_sz, [_i32] * 5),
    "tlaloc_b200_latent_attention": (ctypes.c_int, [_vp, _vp, _i64, _i32, _vp, _vp, _vp, _vp, _vp, _sz] + [_i32] * 10 + [_f32, _vp]),
    "tlaloc_b200_latent_gather": (ctypes.c_int, [_vp, _i64, _i32, _vp, _vp, _i64] + [_i32] * 7 + [_vp]),
    "tlaloc_b200_window_attention_applies": (ctypes.c_int, [_i32] * 3),
    "tlaloc_b200_window_attention": (ctypes.c_int, [_vp, _vp, _i64, _vp, _i64, _vp, _i64, _i64, _vp, _i64] + [_i32] * 12 + [_f32, _vp]),
    "tlaloc_b200_residual_norm": (ctypes.c_int, [_vp, _vp, _i64, _vp, _vp, _vp, _i32, _vp, _vp, _vp, _vp, _i32, _i32, _i32, _f32, _vp]),
    "tlaloc_b200_rotate_rows": (ctypes.c_int, [_vp, _i64, ctypes.POINTER(RotatePart), _i32, _i32, _vp, _vp, _vp, _vp] + [_i32] * 4 + [_vp]),
    "tlaloc_b200_grouped_attention_slices": (ctypes.c_int, [_i32] * 9),
    "tlaloc_b200_grouped_attention": (ctypes.c_int, [_vp, _vp, _i64, _i32, _vp, _vp, _vp, _vp] + [_i32] * 14 + [_f32, _vp]),
    "tlaloc_b200_map_difference": (ctypes.c_int, [_vp, _i32, _vp, _i64, _vp, _i64] + [_i32] * 5 + [_f32, _f32, _f32, _vp]),
    "tlaloc_b200_head_norm_gate": (ctypes.c_int, [_vp, _vp, _i64, _vp, _i64] + [_i32] * 4 + [_f32, _vp]),
    "tlaloc_b200_retention_step": (ctypes.c_int, [_vp, _i64] + [_vp] * 7 + [_i64] + [_i32] * 8 + [_f32, _f32, _vp]),
    "tlaloc_b200_retention_scan": (ctypes.c_int, [_vp, _vp, _i32, _vp, _i32, _i32] + [_vp] * 5 + [_i32] * 5 + [_vp]),
    "tlaloc_b200_retention_chunks_applies": (ctypes.c_int, [_i32] * 2),
    "tlaloc_b200_retention_chunks_scratch_bytes": (_sz, [_i32] * 4),
    "tlaloc_b200_retention_chunks": (ctypes.c_int, [_vp, _vp, _i32, _vp, _i32] + [_vp] * 6 + [_sz] + [_i32] * 5 + [_vp]),
    "tlaloc_b200_moe_route": (ctypes.c_int, [_vp, _i64] + [_vp] * 5 + [_i32] * 3 + [_vp]),
    "tlaloc_b200_gather_rows": (ctypes.c_int, [_vp, _vp, _vp, _i32, _i64, _vp]),
    "tlaloc_b200_peer_alloc": (ctypes.c_int, [_sz, ctypes.POINTER(_vp), ctypes.c_char_p]),
    "tlaloc_b200_peer_open": (ctypes.c_int, [ctypes.c_char_p, ctypes.POINTER(_vp)]),
    "tlaloc_b200_peer_close": (ctypes.c_int, [_vp]),
    "tlaloc_b200_peer_free": (ctypes.c_int, [_vp]),
    "tlaloc_b200_peer_allreduce_f32": (ctypes.c_int, [ctypes.POINTER(_vp), _sz, _sz, _vp, _i32, _i32, _sz, _vp]),
    "tlaloc_b200_peer_allreduce_rmsnorm_f32": (ctypes.c_int, [ctypes.POINTER(_vp), _sz, _sz, _sz, _vp, _vp, _f32, _i32, _i32,
                                                              _i32, _i32, _vp]),
    "tlaloc_b200_peer_reduce_rmsnorm_rows_f32": (ctypes.c_int, [ctypes.POINTER(_vp), _sz, _sz, _sz, _vp, _vp, _vp, _f32, _i32, _i32,
                                                               _i32, _i32, _i32, _vp]),
    "tlaloc_b200_peer_sum_rows_f32": (ctypes.c_int, [ctypes.POINTER(_vp), _sz, _sz, _vp, _vp, _vp, _vp, _vp, _f32, _i32, _i32, _i32, _i32, _vp, _sz, _vp]),
    "TlalocRegisterKernels": (ctypes.c_char_p, [_vp]),
    "tlaloc_b200_ffi_handler": (_vp, [ctypes.c_char_p]),
}


def library_path() -> str:
    return _build.LIB


def declared_symbols() -> list[str]:
    """Every function include/tlaloc_b200.h declares."""
    with open(os.path.join(_build.INCLUDE, "tlaloc_b200.h")) as f:
        text = re.sub(r"/\*.*?\*/", "", f.read(), flags=re.S)
    return sorted(set(re.findall(r"\b(tlaloc_b200_\w+|TlalocRegisterKernels)\s*\(", text)))


def select(subset: str | None) -> None:
    """Before the library is first used: this process needs only the kernels of one of build.SUBSETS."""
    global _subset
    if _lib is None:
        _subset = subset


def lib() -> ctypes.CDLL:
    global _lib
    if _lib is None:
        path = _build.build(subset=_subset)
        if not os.path.exists(path):
            raise RuntimeError(f"{path} is missing: the CUDA extension has not been built (python -m tlaloc_b200.build)")
        loaded = ctypes.CDLL(path)
        for name, (res, args) in _SIGNATURES.items():
            if path != _build.LIB and not hasattr(loaded, name):
                continue  # a kernel outside the subset
            fn = getattr(loaded, name)
            fn.restype, fn.argtypes = res, args
        _lib = loaded
    return _lib


class KernelError(RuntimeError):
    def __init__(self, status: int, message: str):
        super().__init__(message)
        self.status = status


def check(status: int) -> None:
    if status != OK:
        raise KernelError(status, lib().tlaloc_b200_last_error().decode())
