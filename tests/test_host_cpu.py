"""CPU checks of the host side: the library loads and exports what the header declares, the ABI structs match
the headers the reference vendors, the operand parser refuses what the reference refuses."""
import ctypes
import os
import threading
import subprocess
import tempfile

import numpy as np
import pytest

from tlaloc_b200 import _native as N
from tlaloc_b200 import build as B
from tlaloc_b200.attrs import parse_paged_attention

REF_XLA = "/root/reference/triton/third_party/xla"


def test_library_loads_and_exports_every_declared_symbol():
    lib = N.lib()
    names = N.declared_symbols()
    assert "tlaloc_b200_paged_attention" in names and "TlalocRegisterKernels" in names and len(names) >= 17
    for name in names:
        assert hasattr(lib, name), name
        assert name in N._SIGNATURES, f"{name} has no ctypes signature"
    assert lib.tlaloc_b200_abi_version() == 1
    seen = []
    t = threading.Thread(target=lambda: seen.append(lib.tlaloc_b200_last_error()))  # the message is per thread:
    t.start()                                                                        # a new thread has none yet
    t.join()
    assert seen == [b""]


def test_a_subset_of_the_kernels_is_a_library_of_its_own():
    path = B.build(subset="latent", own=True)
    assert os.path.basename(path) == "libtlaloc_latent.so"
    lib = ctypes.CDLL(path)  # every symbol it needs is in it
    for name in ("init", "device_status", "embedding", "argmax", "dense_gemm", "rmsnorm_pair", "latent_kv_write", "rope_interleaved",
                 "latent_attention", "latent_attention_scratch_bytes", "latent_gather", "window_attention", "window_attention_applies"):
        assert hasattr(lib, "tlaloc_b200_" + name), name
    assert not hasattr(lib, "tlaloc_b200_int8_gemm")
    lib = ctypes.CDLL(B.build(subset="mixed", own=True))
    for name in ("init", "device_status", "embedding", "argmax", "dense_gemm", "rmsnorm_pair", "latent_gather", "window_attention", "residual_norm", "rotate_rows",
                 "grouped_attention", "map_difference", "retention_step", "retention_scan", "retention_chunks", "head_norm_gate", "moe_route", "gather_rows"):
        assert hasattr(lib, "tlaloc_b200_" + name), name


def test_dense_and_latent_refusals_need_no_gpu():
    lib = N.lib()
    one, i = ctypes.c_void_p(16), N.INVALID_ARGUMENT
    p = N.DenseProblem(x=16, w=16, y=16, ld_x=8, ld_y=8, k=8, n=8, batch=1, act=0, y_dtype=N.F32)
    call = lambda count=1, dtype=N.BF16, m=1: lib.tlaloc_b200_dense_gemm((N.DenseProblem * 2)(p, p), count, dtype, m, 0, None)
    assert call(count=3) == i and call(dtype=N.S8) == i and call(m=-1) == i and call(m=0) == N.OK
    for field, bad in (("k", 0), ("ld_x", 4), ("ld_y", 4), ("act", 7), ("y_dtype", N.S8), ("x", None), ("batch", 0)):
        was = getattr(p, field)
        setattr(p, field, bad)
        assert call() == i, field
        setattr(p, field, was)
    att = lambda **kw: lib.tlaloc_b200_latent_attention(one, one, kw.get("ld", 56), N.BF16, one, None, one, one, None, 0, kw.get("rows", 1), 3, 48, 8, 9,
                                                        64, 4, kw.get("tables", 1), kw.get("window", 0), 0, 0.1, None)
    assert att(ld=40) == i and att(rows=2) == i and att(window=-1) == i and att(rows=0) == N.OK
    assert lib.tlaloc_b200_window_attention_applies(128, 64, 128) == 1 and lib.tlaloc_b200_window_attention_applies(12, 4, 10) == 0
    win = lambda **kw: lib.tlaloc_b200_window_attention(one, one, 48, one, 8, one, 48, 96, one, 48, N.BF16, kw.get("q", 2), kw.get("k", 2), 0, kw.get("heads", 2),
                                                        kw.get("v_heads", 2), kw.get("maps", 1), 24, 8, 24, 0, kw.get("keep", 0), kw.get("scale", 0.1), None)
    assert win(q=3) == i and win(scale=-1.0) == N.UNSUPPORTED and win(q=0) == N.OK
    assert win(heads=3) == i and win(maps=4) == i and win(v_heads=0) == i and win(keep=-1) == i
    gather = lambda first, keep, count: lib.tlaloc_b200_latent_gather(one, 56, N.BF16, one, one, 56, first, keep, count, 56, 9, 64, 4, None)
    assert gather(200, 0, 100) == i and gather(5, 6, 20) == i and gather(200, 50, 40) == i and gather(200, 50, 107) == i and gather(256, 0, 0) == N.OK


def test_refusals_of_the_mixers_need_no_gpu():
    lib = N.lib()
    one, i = ctypes.c_void_p(16), N.INVALID_ARGUMENT
    assert lib.tlaloc_b200_residual_norm(None, None, 0, None, None, None, 0, one, one, one, one, N.BF16, 1, 8, 1e-5, None) == i
    assert lib.tlaloc_b200_residual_norm(one, None, 0, None, None, None, 2, one, one, one, one, N.BF16, 1, 8, 1e-5, None) == i
    part = N.RotatePart(out=16, out_ld=16, out_head_ld=8, first=0, heads=2, dim=8, padded=8, rotate=1, by_slot=0, scale=1.0)
    rotate = lambda ld=16, dims=8, slots=None: lib.tlaloc_b200_rotate_rows(one, ld, ctypes.byref(part), 1, N.BF16, one, one, one, slots, 0, dims, 4, 4, None)
    assert rotate() == N.OK and rotate(ld=15) == i and rotate(dims=10) == i and rotate(dims=7) == i
    part.by_slot = 1
    assert rotate() == i
    att = lambda **kw: lib.tlaloc_b200_grouped_attention(one, one, kw.get("ld", 96), N.BF16, one, None, one, one, kw.get("slices", 1), kw.get("rows", 0), kw.get("heads", 8),
                                                         2, 2, 16, 16, kw.get("v_first", 64), 9, 64, 4, 1, kw.get("window", 0), kw.get("keep", 0), 0.1, None)
    assert att() == N.OK and att(ld=95) == i and att(heads=6) == i and att(v_first=63) == i and att(window=-1) == i and att(keep=-1) == i and att(slices=0) == i
    assert lib.tlaloc_b200_grouped_attention_slices(4, 8, 2, 2, 24, 16, 64, N.BF16, 4096) == 1  # not the tensor-core kernel's sizes
    assert lib.tlaloc_b200_map_difference(one, -1, None, 0, one, 16, N.BF16, 1, 2, 8, 8, 0.1, 0.5, 1e-5, None) == i
    assert lib.tlaloc_b200_map_difference(one, 0, None, 0, one, 15, N.BF16, 1, 2, 8, 8, 0.1, 0.5, 1e-5, None) == i
    assert lib.tlaloc_b200_head_norm_gate(one, one, 16, one, 15, N.BF16, 1, 2, 8, 1e-5, None) == i
    step = lambda **kw: lib.tlaloc_b200_retention_step(one, kw.get("ld", 64), one, one, one, one, one, one, one, 16, N.BF16, kw.get("rows", 0), 2, kw.get("dim", 8), 8,
                                                       kw.get("rot", 8), 3, 4, 0.3, 1e-5, None)
    assert step() == N.OK and step(ld=63) == i and step(rot=10) == i and step(rows=-1) == i and step(dim=520, ld=9999) == N.UNSUPPORTED
    assert lib.tlaloc_b200_retention_scan(one, one, 7, one, 8, N.BF16, one, one, one, one, one, 4, 2, 8, 8, 3, None) == i
    chunks = lambda dim=24, dim_ld=32, tokens=4: lib.tlaloc_b200_retention_chunks(one, one, dim_ld, one, 16, one, one, one, one, one, None, 0, tokens, 2, dim, 8, 3, None)
    assert chunks(dim_ld=24) == i and chunks(dim=257, dim_ld=272) == N.UNSUPPORTED and chunks(tokens=0) == N.OK and chunks(tokens=2048) == i  # no scratch
    assert lib.tlaloc_b200_moe_route(one, 4, one, one, one, one, one, 3, 5, 2, None) == i and lib.tlaloc_b200_moe_route(one, 8, one, one, one, one, one, 3, 5, 6, None) == i
    assert lib.tlaloc_b200_gather_rows(one, one, one, 1, 3, None) == i
    g = N.DenseProblem(x=16, w=16, y=16, ld_x=8, ld_y=16, k=8, n=32, batch=1, act=N.ACT_SILU_MUL, y_dtype=N.F32)
    dense = lambda *ps: lib.tlaloc_b200_dense_gemm((N.DenseProblem * len(ps))(*ps), len(ps), N.BF16, 0, 0, None)
    assert dense(g) == N.OK
    g.n = 40
    assert dense(g) == i  # gate and factor come in blocks of 16
    g.n, g.bias = 32, 16
    assert dense(g) == i
    g.bias, g.row_offsets = None, 16
    assert dense(g) == N.OK and dense(g, g) == i  # a grouped projection is the last of a call


def test_argument_refusals_need_no_gpu():
    lib = N.lib()
    # a null pointer, a bad dtype and a bad shape are refused before any CUDA call
    rc = lib.tlaloc_b200_paged_attention(None, N.F32, None, None, N.F32, None, None, None, 0, None, N.F32, None, None, 1,
                                         1, 1, 1, 1, 1, 1, 1, 1, 1.0, 0, None)
    assert rc == N.INVALID_ARGUMENT and b"null" in lib.tlaloc_b200_last_error()
    one = ctypes.c_void_p(16)
    rc = lib.tlaloc_b200_paged_attention(one, N.F32, one, one, N.F32, one, one, None, 0, one, N.F32, None, one, 1,
                                         3, 4, 8, 6, 2, 3, 3, 2, 0.5, 0, None)  # 4 heads over 3 kv heads
    assert rc == N.INVALID_ARGUMENT and b"multiple of numKvHeads" in lib.tlaloc_b200_last_error()
    rc = lib.tlaloc_b200_paged_attention(one, N.F32, one, one, N.F32, one, one, None, 0, one, N.F32, None, one, 1,
                                         3, 4, 8, 6, 2, 2, 3, 2, 0.5, 0, None)  # 3 rows over 2 tables
    assert rc == N.INVALID_ARGUMENT and b"one per row" in lib.tlaloc_b200_last_error()
    rc = lib.tlaloc_b200_paged_attention(one, N.S8, one, one, N.F32, one, one, None, 0, one, N.F32, None, one, 1,
                                         2, 4, 8, 6, 2, 2, 3, 2, 0.5, 0, None)
    assert rc == N.INVALID_ARGUMENT and b"f32 or bf16" in lib.tlaloc_b200_last_error()
    rc = lib.tlaloc_b200_int8_gemm(one, N.F32, one, one, None, one, N.F32, None, 0, 0, 8, 8, 0, None)
    assert rc == N.INVALID_ARGUMENT
    rc = lib.tlaloc_b200_rope_kv_write(one, one, one, one, one, one, one, one, N.F32, one, one, N.F32, 1, 4, 2, 3, 8, 8, 12, 6, 6, None)
    assert rc == N.INVALID_ARGUMENT and b"odd" in lib.tlaloc_b200_last_error()
    assert lib.tlaloc_b200_paged_attention_splits(32, 8, 32, 512, 16) == 32
    assert lib.tlaloc_b200_paged_attention_scratch_bytes(32, 32, 128, 32) == 32 * 32 * 32 * 130 * 4
    assert lib.tlaloc_b200_ffi_handler(b"tlaloc_paged_attention") and lib.tlaloc_b200_ffi_handler(b"nope") is None


class _T:
    def __init__(self, shape, dtype="float32"):
        self.shape, self.dtype = shape, dtype


def test_parser_refuses_what_the_reference_refuses():
    """ir/src/commonTest/.../PagedAttentionTest.kt:518-567 and PagedAttentionAttrs.kt:145-286."""
    q, k = _T((2, 4, 3)), _T((6, 2, 2, 3))
    t, l = _T((2, 3), "int32"), _T((2,), "int32")
    p = parse_paged_attention(q, k, k, t, l, scale=0.5)
    assert (p.group, p.rows_per_table, p.max_context_len, p.first_live(5)) == (2, 1, 6, 0)
    assert parse_paged_attention(q, k, k, t, l, scale=0.5, sliding_window=2).first_live(5) == 3
    p3 = parse_paged_attention(_T((6, 4, 3)), k, k, t, _T((6,), "int32"), scale=0.5)
    assert p3.rows_per_table == 3 and p3.table_of(5) == 1

    def refused(match, *a, **kw):
        with pytest.raises(ValueError, match=match):
            parse_paged_attention(*a, **kw)

    refused("sliding_window", q, k, k, t, l, scale=0.5, sliding_window=0)
    refused("one per row", _T((3, 4, 3)), k, k, t, _T((3,), "int32"), scale=0.5)
    refused("scale", q, k, k, t, l, scale=None)
    refused("finite", q, k, k, t, l, scale=float("inf"))
    refused("refused by name", q, k, k, t, l, scale=0.5, block_size=2)
    refused("refused by name", q, k, k, t, l, scale=0.5, numKvHeads=2)
    refused("rank-3", _T((2, 12)), k, k, t, l, scale=0.5)
    refused("valueCache shape", q, k, _T((6, 2, 2, 4)), t, l, scale=0.5)
    refused("integer tensor", q, k, k, _T((2, 3), "float32"), l, scale=0.5)
    refused("multiple of numKvHeads", _T((2, 3, 3)), k, k, t, l, scale=0.5)
    refused("keep has 4 chunks", q, k, k, t, l, scale=0.5, keep=_T((2, 4), "int32"))
    refused("return_lse", q, k, k, t, l, scale=0.5, return_lse=True, sliding_window=2)
    assert parse_paged_attention(q, k, k, t, l, scale=0.5, keep=_T((2, 3), "int32")).keep_chunk == 2


@pytest.mark.skipif(not os.path.isdir(REF_XLA), reason="the XLA headers the reference vendors are not mounted")
def test_abi_structs_match_the_vendored_xla_headers():
    """Every offset and size tlaloc_b200/csrc/xla_abi.h relies on, against xla/ffi/api/c_api.h and the PJRT headers."""
    checks = [
        ("AbiFfiCallFrame", "XLA_FFI_CallFrame", ["struct_size", "extension_start", "api", "ctx", "stage", "args", "rets", "attrs", "future"]),
        ("AbiFfiBuffer", "XLA_FFI_Buffer", ["struct_size", "extension_start", "dtype", "data", "rank", "dims"]),
        ("AbiFfiArgs", "XLA_FFI_Args", ["struct_size", "extension_start", "size", "types", ("values", "args")]),
        ("AbiFfiArgs", "XLA_FFI_Rets", ["struct_size", "extension_start", "size", "types", ("values", "rets")]),
        ("AbiFfiAttrs", "XLA_FFI_Attrs", ["struct_size", "extension_start", "size", "types", "names", ("values", "attrs")]),
        ("AbiFfiExtensionBase", "XLA_FFI_InternalExtension", ["struct_size", "type", "next"]),
        ("AbiFfiMetadata", "XLA_FFI_Metadata", ["struct_size", "api_version", "traits", "state_type_id"]),
        ("AbiFfiMetadataExtension", "XLA_FFI_Metadata_Extension", [("base", "extension_base"), "metadata"]),
        ("AbiFfiApiVersion", "XLA_FFI_Api_Version", ["struct_size", "extension_start", "major_version", "minor_version"]),
        ("AbiFfiScalar", "XLA_FFI_Scalar", ["dtype", "value"]),
        ("AbiFfiByteSpan", "XLA_FFI_ByteSpan", ["ptr", "len"]),
        ("AbiFfiErrorCreateArgs", "XLA_FFI_Error_Create_Args", ["struct_size", "extension_start", "message", "errc"]),
        ("AbiFfiStreamGetArgs", "XLA_FFI_Stream_Get_Args", ["struct_size", "extension_start", "ctx", "stream"]),
        ("AbiFfiApi", "XLA_FFI_Api", ["struct_size", "extension_start", "api_version", "internal_api",
                                       ("error_create", "XLA_FFI_Error_Create"), ("error_destroy", "XLA_FFI_Error_Destroy"),
                                       ("stream_get", "XLA_FFI_Stream_Get")]),
        ("AbiPjrtExtensionBase", "PJRT_Extension_Base", ["struct_size", "type", "next"]),
        ("AbiPjrtApiHead", "PJRT_Api", ["struct_size", "extension_start", "pjrt_api_version",
                                         ("error_destroy", "PJRT_Error_Destroy"), ("error_message", "PJRT_Error_Message")]),
        ("AbiPjrtErrorMessageArgs", "PJRT_Error_Message_Args", ["struct_size", "extension_start", "error", "message", "message_size"]),
        ("AbiPjrtErrorDestroyArgs", "PJRT_Error_Destroy_Args", ["struct_size", "extension_start", "error"]),
        ("AbiPjrtGpuRegisterCustomCallArgs", "PJRT_Gpu_Register_Custom_Call_Args",
         ["struct_size", "function_name", "function_name_size", "api_version", "handler_instantiate", "handler_prepare",
          "handler_initialize", "handler_execute", "traits"]),
        ("AbiPjrtGpuCustomCall", "PJRT_Gpu_Custom_Call", ["base", "custom_call", "custom_call_handles_traits"]),
    ]
    lines = ['#include <cstddef>', '#include "xla/ffi/api/c_api.h"', '#include "xla/pjrt/c/pjrt_c_api.h"',
             '#include "xla/pjrt/c/pjrt_c_api_gpu_extension.h"', f'#include "{B.CSRC}/xla_abi.h"']
    for mine, theirs, fields in checks:
        for f in fields:
            a, b = f if isinstance(f, tuple) else (f, f)
            lines.append(f'static_assert(offsetof({mine}, {a}) == offsetof({theirs}, {b}), "{mine}.{a}");')
            lines.append(f'static_assert(sizeof((({mine}*)0)->{a}) == sizeof((({theirs}*)0)->{b}), "{mine}.{a} size");')
    consts = [("kAbiFfiExtensionMetadata", "XLA_FFI_Extension_Metadata"), ("kAbiFfiInitialize", "XLA_FFI_ExecutionStage_INITIALIZE"),
              ("kAbiFfiExecute", "XLA_FFI_ExecutionStage_EXECUTE"), ("kAbiFfiInvalidArgument", "XLA_FFI_Error_Code_INVALID_ARGUMENT"),
              ("kAbiFfiInternal", "XLA_FFI_Error_Code_INTERNAL"), ("kAbiFfiAttrScalar", "XLA_FFI_AttrType_SCALAR"),
              ("kAbiFfiApiMajor", "XLA_FFI_API_MAJOR"), ("kAbiFfiApiMinor", "XLA_FFI_API_MINOR"),
              ("kAbiFfiTraitCommandBufferCompatible", "XLA_FFI_HANDLER_TRAITS_COMMAND_BUFFER_COMPATIBLE"),
              ("kAbiPjrtExtensionGpuCustomCall", "PJRT_Extension_Type_Gpu_Custom_Call"),
              ("TLALOC_B200_F32", "XLA_FFI_DataType_F32"), ("TLALOC_B200_BF16", "XLA_FFI_DataType_BF16"),
              ("TLALOC_B200_S8", "XLA_FFI_DataType_S8"), ("TLALOC_B200_S32", "XLA_FFI_DataType_S32"),
              ("TLALOC_ABI_SIZE_THROUGH(AbiFfiErrorCreateArgs, errc)", "XLA_FFI_Error_Create_Args_STRUCT_SIZE"),
              ("TLALOC_ABI_SIZE_THROUGH(AbiFfiStreamGetArgs, stream)", "XLA_FFI_Stream_Get_Args_STRUCT_SIZE"),
              ("TLALOC_ABI_SIZE_THROUGH(AbiPjrtGpuRegisterCustomCallArgs, traits)", "PJRT_Gpu_Register_Custom_Call_Args_STRUCT_SIZE"),
              ("TLALOC_ABI_SIZE_THROUGH(AbiPjrtErrorMessageArgs, message_size)", "PJRT_Error_Message_Args_STRUCT_SIZE"),
              ("TLALOC_ABI_SIZE_THROUGH(AbiPjrtErrorDestroyArgs, error)", "PJRT_Error_Destroy_Args_STRUCT_SIZE")]
    lines.append(f'#include "{B.INCLUDE}/tlaloc_b200.h"')
    for mine, theirs in consts:
        lines.append(f'static_assert((long)({mine}) == (long)({theirs}), "{theirs}");')
    lines.append("int main() { return 0; }")
    with tempfile.TemporaryDirectory() as d:
        src = os.path.join(d, "abi_check.cc")
        with open(src, "w") as f:
            f.write("\n".join(lines))
        r = subprocess.run(["g++", "-std=c++17", "-fsyntax-only", "-I", REF_XLA, src], capture_output=True, text=True)
        assert r.returncode == 0, r.stderr[-3000:]


def test_peer_sum_refuses_bad_arguments_before_touching_the_gpu():
    """The tensor-parallel sum validates on the host first; world 1 is a no-op (no device is needed for either)."""
    lib = N.lib()
    bases = (ctypes.c_void_p * 2)(0x1000, 0x2000)
    state = ctypes.c_void_p(0x3000)
    call = lib.tlaloc_b200_peer_allreduce_f32
    assert call(bases, 0, 0, state, 0, 9, 4, None) == N.INVALID_ARGUMENT and b"world 9" in lib.tlaloc_b200_last_error()
    assert call(bases, 0, 0, state, 2, 2, 4, None) == N.INVALID_ARGUMENT and b"rank 2" in lib.tlaloc_b200_last_error()
    assert call(bases, 0, 0, state, 0, 2, 6, None) == N.INVALID_ARGUMENT  # count not a multiple of 4
    assert call(bases, 8, 0, state, 0, 2, 4, None) == N.INVALID_ARGUMENT  # values not 16-byte aligned
    assert call(None, 0, 0, state, 0, 2, 4, None) == N.INVALID_ARGUMENT
    misaligned = (ctypes.c_void_p * 2)(0x1000, 0x2004)
    assert call(misaligned, 0, 0, state, 0, 2, 4, None) == N.INVALID_ARGUMENT and b"rank 1" in lib.tlaloc_b200_last_error()
    assert call(bases, 0, 0, state, 0, 1, 4, None) == N.OK  # one rank: nothing to exchange, nothing launched
    assert call(bases, 0, 0, state, 0, 2, 0, None) == N.OK

    from tlaloc_b200.peer import PeerBuffers

    with pytest.raises(ValueError):
        PeerBuffers([(4, 4)], rank=0, world=9)


def test_fused_peer_sum_and_norm_refuses_bad_shapes_before_touching_the_gpu():
    lib = N.lib()
    bases = (ctypes.c_void_p * 2)(0x1000, 0x2000)
    state = ctypes.c_void_p(0x3000)
    call = lib.tlaloc_b200_peer_allreduce_rmsnorm_f32
    assert call(bases, 0, 4096, 8192, state, None, 1e-5, 0, 1, 4, 256, None) == N.INVALID_ARGUMENT  # one rank: use rmsnorm
    assert call(bases, 0, 4096, 8192, state, None, 1e-5, 0, 2, 3, 256, None) == N.INVALID_ARGUMENT  # rows do not divide
    assert b"3 rows" in lib.tlaloc_b200_last_error()
    assert call(bases, 0, 4096, 8192, state, None, 1e-5, 0, 2, 4, 250, None) == N.INVALID_ARGUMENT  # cols not a multiple of 16
    assert call(bases, 0, 4096, 8192, state, None, 1e-5, 0, 2, 4, 65536, None) == N.INVALID_ARGUMENT  # a row too long for registers
    assert call(bases, 0, 4100, 8192, state, None, 1e-5, 0, 2, 4, 256, None) == N.INVALID_ARGUMENT  # norm region misaligned
    assert call(bases, 0, 4096, 8192, state, ctypes.c_void_p(0x4004), 1e-5, 0, 2, 4, 256, None) == N.INVALID_ARGUMENT  # gain misaligned
