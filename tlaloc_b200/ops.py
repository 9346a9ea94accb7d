"""The hot-path operators on torch CUDA tensors, through the C ABI.

PyTorch is plumbing here (device memory, the current stream); every operator is one call into
libtlaloc_kernels.so with raw device pointers, enqueued on torch's current stream.  There is no CPU path:
a tensor that is not on a CUDA device is refused.
"""
from __future__ import annotations

import torch

from . import _native as N
from .attrs import PagedAttentionShape, parse_paged_attention

_DT = {torch.float32: N.F32, torch.bfloat16: N.BF16, torch.int8: N.S8, torch.int32: N.S32, torch.float8_e4m3fn: N.F8E4M3FN}


def _dt(t: torch.Tensor) -> int:
    try:
        return _DT[t.dtype]
    except KeyError:
        raise TypeError(f"unsupported dtype {t.dtype}") from None


def _dev(*ts) -> None:
    for t in ts:
        if t is not None and (not t.is_cuda or not t.is_contiguous()):
            raise ValueError("operands must be contiguous CUDA tensors (there is no CPU path)")


def _out(name: str, t, shape, dtypes, like: torch.Tensor) -> None:
    """A caller-supplied result or scratch tensor is written through its raw pointer: refuse one that is not exactly
    the contiguous CUDA tensor of that shape the kernel will write."""
    if t is None:
        return
    if not isinstance(dtypes, (tuple, list)):
        dtypes = (dtypes,)
    if (not t.is_cuda or not t.is_contiguous() or t.device != like.device or t.dtype not in dtypes
            or (shape is not None and tuple(t.shape) != tuple(shape))):
        want = "x".join(str(d) for d in shape) if shape is not None else "any shape"
        raise ValueError(f"{name} must be a contiguous {'/'.join(str(d) for d in dtypes)} tensor [{want}] on {like.device}, "
                         f"got {t.dtype} {tuple(t.shape)} on {t.device}")


def _ptr(t):
    return None if t is None else t.data_ptr()


def _stream(t: torch.Tensor) -> int:
    """The current stream of the tensor's own device (not of whichever device happens to be current)."""
    return torch.cuda.current_stream(t.device).cuda_stream


def init() -> None:
    """Kernel set-up for the current CUDA device (call once per device, before any graph capture)."""
    N.check(N.lib().tlaloc_b200_init())


def set_order_faithful(on: bool) -> bool:
    """Parity mode of the whole library (tlaloc_b200_set_order_faithful); returns the previous setting."""
    return bool(N.lib().tlaloc_b200_set_order_faithful(1 if on else 0))


def paged_attention_scratch(shape: PagedAttentionShape, device, splits: int | None = None) -> torch.Tensor:
    """The f32 scratch [S, R, H, D + 2] a call of this shape wants (S as the reference's emitter sizes it)."""
    lib = N.lib()
    if splits is None:
        splits = lib.tlaloc_b200_paged_attention_splits(shape.num_seqs, shape.num_kv_heads, shape.num_tables,
                                                        shape.max_blocks_per_seq, shape.block_size)
    return torch.empty((splits, shape.num_seqs, shape.num_heads, shape.head_dim + 2), dtype=torch.float32, device=device)


def paged_attention(query, key_cache, value_cache, block_tables, seq_lens, *, scale, sliding_window=None, keep=None,
                    return_lse=False, out=None, scratch=None):
    """PAGED_ATTENTION: operands and attrs as ir/.../PagedAttentionAttrs.kt; see include/tlaloc_b200.h."""
    p = parse_paged_attention(query, key_cache, value_cache, block_tables, seq_lens, scale=scale,
                              sliding_window=sliding_window, keep=keep, layer="tlaloc_b200.ops")
    _dev(query, key_cache, value_cache, block_tables, seq_lens, keep)
    if block_tables.dtype != torch.int32 or seq_lens.dtype != torch.int32 or (keep is not None and keep.dtype != torch.int32):
        raise TypeError("PAGED_ATTENTION: the kernels read blockTables, seqLens and keep as int32")
    if out is None:
        out = torch.empty_like(query)
    if scratch is None:
        scratch = paged_attention_scratch(p, query.device)
    _out("PAGED_ATTENTION out", out, (p.num_seqs, p.num_heads, p.head_dim), (torch.float32, torch.bfloat16), query)
    if scratch.dim() != 4 or scratch.shape[0] < 1:
        raise ValueError("PAGED_ATTENTION scratch must be f32 [S, R, H, D + 2] with S >= 1")
    _out("PAGED_ATTENTION scratch", scratch, (scratch.shape[0], p.num_seqs, p.num_heads, p.head_dim + 2), torch.float32, query)
    lse = torch.empty((p.num_seqs, p.num_heads), dtype=torch.float32, device=query.device) if return_lse else None
    N.check(N.lib().tlaloc_b200_paged_attention(
        _ptr(query), _dt(query), _ptr(key_cache), _ptr(value_cache), _dt(key_cache), _ptr(block_tables),
        _ptr(seq_lens), _ptr(keep), 0 if keep is None else keep.shape[1], _ptr(out), _dt(out), _ptr(lse),
        _ptr(scratch), scratch.shape[0], p.num_seqs, p.num_heads, p.head_dim, p.num_blocks, p.block_size,
        p.num_kv_heads, p.max_blocks_per_seq, p.num_tables, float(scale), int(sliding_window or 0), _stream(query)))
    return (out, lse) if return_lse else out


def kv_cache_write(pool, new_kv, slot_mapping):
    """KV_CACHE_WRITE in place: pool [P, bs, Hkv, D], new_kv [T, Hkv, D], slot_mapping i32 [T]."""
    _dev(pool, new_kv, slot_mapping)
    P, bs, Hkv, D = pool.shape
    T = slot_mapping.shape[0]
    if new_kv.numel() != T * Hkv * D:
        raise ValueError(f"KV_CACHE_WRITE: newKv must be [T, {Hkv}, {D}] for the pool, got {tuple(new_kv.shape)}")
    N.check(N.lib().tlaloc_b200_kv_cache_write(_ptr(pool), _dt(pool), _ptr(new_kv), _dt(new_kv), _ptr(slot_mapping), T,
                                               Hkv * D, P * bs, _stream(pool)))
    return pool


def int8_gemm(x, codes, scales, *, residual=None, out=None, out_dtype=torch.float32, exact=False, x_f32_exact=False,
              scratch=None, weights_const=False, i8_mma=False, x_planes=False):
    """y = (cast(x) @ cast(codes)) * scales (+ residual): x [M, K], codes int8 [K, N] (in, out), scales f32 [N].
    `weights_const`: no kernel queued just before this call writes codes or scales (true of a loaded model).
    `i8_mma`: 17 to 128 rows take the int8 tensor-core kernel (codes straight to the tensor core, activations as 16-bit
    fixed point per row, exact int32 sums) instead of the bf16 one (f32 accumulation of exact products).
    `x_planes`: `scratch` already holds x's activation planes (rmsnorm(..., planes=scratch) wrote them)."""
    _dev(x, codes, scales, residual)
    M, K = x.shape
    K2, Nn = codes.shape
    if K2 != K or codes.dtype != torch.int8 or (scales is not None and tuple(scales.shape) != (Nn,)):
        raise ValueError(f"INT8_PROJ: x [M, K] x codes int8 [K, N] with scales [N]; got {tuple(x.shape)}, {tuple(codes.shape)}")
    if out is None:
        out = torch.empty((M, Nn), dtype=out_dtype, device=x.device)
    _out("INT8_PROJ out", out, (M, Nn), (torch.float32, torch.bfloat16), x)
    _out("INT8_PROJ residual", residual, (M, Nn), torch.float32, x)
    # an f32 x is cast to bf16 in the scratch; the int8 tensor-core kernel leaves the activations' int8 planes there
    if scratch is None and not exact and (x.dtype == torch.float32 or (i8_mma and 17 <= M <= 128)):
        scratch = torch.empty((N.lib().tlaloc_b200_int8_gemm_scratch_bytes(M, K, Nn) + 3) // 4, dtype=torch.float32,
                              device=x.device)
    _out("INT8_PROJ scratch", scratch, None, torch.float32, x)
    flags = ((N.GEMM_EXACT if exact else 0) | (N.GEMM_X_F32_EXACT if x_f32_exact else 0)
             | (N.GEMM_WEIGHTS_CONST if weights_const else 0) | (N.GEMM_I8_MMA if i8_mma else 0)
             | (N.GEMM_X_PLANES if x_planes else 0))
    N.check(N.lib().tlaloc_b200_int8_gemm(_ptr(x), _dt(x), _ptr(codes), _ptr(scales), _ptr(residual), _ptr(out), _dt(out),
                                          _ptr(scratch), 0 if scratch is None else scratch.numel() * 4, M, K, Nn, flags,
                                          _stream(x)))
    return out


def int8_gemm_swiglu(x, codes, scales, *, out=None, out_dtype=torch.bfloat16, exact=False, scratch=None, weights_const=False,
                     i8_mma=False, x_planes=False):
    """silu(x @ gate) * (x @ up) with gate and up interleaved in `codes` [K, 2F] in column blocks of 128 + 128
    (sharding.interleave_gate_up); returns [M, F]."""
    _dev(x, codes, scales)
    M, K = x.shape
    K2, Nn = codes.shape
    if K2 != K or codes.dtype != torch.int8 or Nn % 256 or (scales is not None and tuple(scales.shape) != (Nn,)):
        raise ValueError(f"INT8_PROJ_SWIGLU: x [M, K] x codes int8 [K, 2F] (2F a multiple of 256) with scales [2F]; got "
                         f"{tuple(x.shape)}, {tuple(codes.shape)}")
    if out is None:
        out = torch.empty((M, Nn // 2), dtype=out_dtype, device=x.device)
    _out("INT8_PROJ_SWIGLU out", out, (M, Nn // 2), (torch.float32, torch.bfloat16), x)
    if scratch is None and not exact and (x.dtype == torch.float32 or (i8_mma and 17 <= M <= 128)):
        scratch = torch.empty((N.lib().tlaloc_b200_int8_gemm_scratch_bytes(M, K, Nn) + 3) // 4, dtype=torch.float32, device=x.device)
    _out("INT8_PROJ_SWIGLU scratch", scratch, None, torch.float32, x)
    flags = ((N.GEMM_EXACT if exact else 0) | (N.GEMM_WEIGHTS_CONST if weights_const else 0) | (N.GEMM_I8_MMA if i8_mma else 0)
             | (N.GEMM_X_PLANES if x_planes else 0))
    N.check(N.lib().tlaloc_b200_int8_gemm_swiglu(_ptr(x), _dt(x), _ptr(codes), _ptr(scales), _ptr(out), _dt(out), _ptr(scratch),
                                                 0 if scratch is None else scratch.numel() * 4, M, K, Nn, flags, _stream(x)))
    return out


def int8_gemm_scratch_bytes(m: int, k: int, n: int) -> int:
    return int(N.lib().tlaloc_b200_int8_gemm_scratch_bytes(m, k, n))


def dense_gemm_exact(x, w, *, x_f32_exact=False):
    """The interpreter's MATMUL order over an unquantized weight w [K, N]; returns f32 [M, N]."""
    _dev(x, w)
    M, K = x.shape
    out = torch.empty((M, w.shape[1]), dtype=torch.float32, device=x.device)
    N.check(N.lib().tlaloc_b200_dense_gemm_exact(_ptr(x), _dt(x), _ptr(w), _dt(w), _ptr(out), M, K, w.shape[1],
                                                 N.GEMM_X_F32_EXACT if x_f32_exact else 0, _stream(x)))
    return out


def embedding(table, ids, *, out=None):
    _dev(table, ids)
    ids = ids.reshape(-1)
    if out is None:
        out = torch.empty((ids.shape[0], table.shape[1]), dtype=torch.float32, device=table.device)
    _out("EMBEDDING out", out, (ids.shape[0], table.shape[1]), torch.float32, table)
    N.check(N.lib().tlaloc_b200_embedding(_ptr(table), _dt(table), _ptr(ids), _ptr(out), ids.shape[0], table.shape[0],
                                          table.shape[1], _stream(table)))
    return out


def rmsnorm(x, gain, eps, *, out=None, out_dtype=torch.float32, planes=None):
    """x * rsqrt(mean(x^2) + eps) * gain.  `planes` (an f32 scratch of int8_gemm_scratch_bytes(rows, n, 0) bytes; out must
    be bf16, n a multiple of 16) also receives the normalised rows as the activation planes of the int8 tensor-core
    projection that reads `out`: call that projection with the same scratch and x_planes=True."""
    _dev(x, gain)
    rows, n = x.shape
    if out is None:
        out = torch.empty((rows, n), dtype=torch.bfloat16 if planes is not None else out_dtype, device=x.device)
    _out("RMSNORM out", out, (rows, n), (torch.float32, torch.bfloat16), x)
    if planes is not None:
        _out("RMSNORM planes", planes, None, torch.float32, x)
        if out.dtype != torch.bfloat16 or planes.numel() * 4 < int8_gemm_scratch_bytes(rows, n, 0):
            raise ValueError("RMSNORM: planes need a bf16 out and int8_gemm_scratch_bytes(rows, n, 0) bytes")
        N.check(N.lib().tlaloc_b200_rmsnorm_planes(_ptr(x), _ptr(gain), _ptr(out), _ptr(planes), planes.numel() * 4, rows, n, float(eps), _stream(x)))
        return out
    N.check(N.lib().tlaloc_b200_rmsnorm(_ptr(x), _ptr(gain), _ptr(out), _dt(out), rows, n, float(eps), _stream(x)))
    return out


def rope_kv_write(q, k, v, positions, cos_table, sin_table, slot_mapping, key_cache, value_cache, *, q_out=None,
                  q_dtype=torch.float32):
    """RoPE on q [T,H,hd] and k [T,Hkv,hd], then K/V rows into the pools at slot_mapping; returns rotated q."""
    _dev(positions, cos_table, sin_table, slot_mapping, key_cache, value_cache)
    for t in (q, k, v):
        if not t.is_cuda or t.dtype != torch.float32 or t.stride(2) != 1 or t.stride(1) != t.shape[2]:
            raise ValueError("ROPE_KV_WRITE: q, k and v must be f32 CUDA tensors [T, heads, hd] with dense heads")
    T, H, hd = q.shape
    Hkv = k.shape[1]
    P, bs = key_cache.shape[0], key_cache.shape[1]
    if q_out is None:
        q_out = torch.empty((T, H, hd), dtype=q_dtype, device=q.device)
    _out("ROPE_KV_WRITE q_out", q_out, (T, H, hd), (torch.float32, torch.bfloat16), q)
    N.check(N.lib().tlaloc_b200_rope_kv_write(_ptr(q), _ptr(k), _ptr(v), _ptr(positions), _ptr(cos_table), _ptr(sin_table),
                                              _ptr(slot_mapping), _ptr(q_out), _dt(q_out), _ptr(key_cache),
                                              _ptr(value_cache), _dt(key_cache), T, H, Hkv, hd, P * bs,
                                              cos_table.shape[0], q.stride(0), k.stride(0), v.stride(0), _stream(q)))
    return q_out


def swiglu(gate, up, *, out=None, out_dtype=torch.float32):
    """silu(gate) * up; gate and up may be column slices of one [rows, ld] matrix (a fused gate|up projection)."""
    if not gate.is_cuda or gate.stride(1) != 1 or up.stride(1) != 1 or gate.stride(0) != up.stride(0):
        raise ValueError("SWIGLU: gate and up must be CUDA row-major views with the same row stride")
    rows, n = gate.shape
    if out is None:
        out = torch.empty((rows, n), dtype=out_dtype, device=gate.device)
    _out("SWIGLU out", out, (rows, n), (torch.float32, torch.bfloat16), gate)
    N.check(N.lib().tlaloc_b200_swiglu(_ptr(gate), _ptr(up), gate.stride(0), _ptr(out), _dt(out), rows, n, _stream(gate)))
    return out


def argmax(logits, out=None):
    _dev(logits)
    rows, n = logits.shape
    if out is None:
        out = torch.empty((rows,), dtype=torch.int32, device=logits.device)
    _out("ARGMAX out", out, (rows,), torch.int32, logits)
    N.check(N.lib().tlaloc_b200_argmax(_ptr(logits), _ptr(out), rows, n, _stream(logits)))
    return out


# ---------------------------------------------------------------------- unquantized projections, latent attention


GATED = (N.ACT_SILU_MUL, N.ACT_GELU_TANH_MUL)


def dense(x, w, out, *, bias=None, residual=None, act=N.ACT_NONE) -> N.DenseProblem:
    """One projection out = act(x @ w.T + bias) + residual for `dense_gemm`.  x [M, K], w [N, K], out [M, N]; or a batch
    of them (the heads of a layer): x [B, M, K], w [B, N, K], out [B, M, N].  x, out and residual may be strided views whose
    last dimension is dense; w is contiguous.  A gated act (see interleave_gate) leaves out [M, N / 2]."""
    batched = w.dim() == 3
    for name, t in (("x", x), ("out", out)) + ((("residual", residual),) if residual is not None else ()):
        if not t.is_cuda or t.stride(-1) != 1 or t.dim() != w.dim():
            raise ValueError(f"DENSE_PROJ {name}: a CUDA tensor of rank {w.dim()} with a dense last dimension is needed")
    _dev(w, bias)
    b, n, k = w.shape if batched else (1, *w.shape)
    m = x.shape[-2]
    if x.shape[-1] != k or tuple(out.shape[-2:]) != (m, n // 2 if act in GATED else n) or (batched and (x.shape[0] != b or out.shape[0] != b)) or x.dtype != w.dtype:
        raise ValueError(f"DENSE_PROJ: x {tuple(x.shape)} {x.dtype}, w {tuple(w.shape)} {w.dtype}, out {tuple(out.shape)} do not fit")
    if (bias is not None and (bias.dtype != torch.float32 or tuple(bias.shape) != (n,))) or (
            residual is not None and (residual.dtype != torch.float32 or tuple(residual.shape) != (m, n))):
        raise ValueError(f"DENSE_PROJ: bias is f32 [{n}], residual f32 [{m}, {n}]")
    p = N.DenseProblem(x=_ptr(x), w=_ptr(w), bias=_ptr(bias), residual=_ptr(residual), y=_ptr(out), ld_x=x.stride(-2),
                       ld_res=residual.stride(-2) if residual is not None else 0, ld_y=out.stride(-2),
                       batch_x=x.stride(0) if batched else 0, batch_w=n * k, batch_y=out.stride(0) if batched else 0,
                       k=k, n=n, batch=b, act=act, y_dtype=_dt(out))
    p.rows, p.like = m, x
    return p


def grouped_dense(x, w, out, row_offsets, *, act=N.ACT_NONE) -> N.DenseProblem:
    """The projections of a batch of weights w [B, N, K], each applied to its own rows [row_offsets[b], row_offsets[b + 1]) of x [M, K]
    -> out [M, N] (N / 2 for a gated act): the last problem of a `dense_gemm` call."""
    _dev(w, row_offsets)
    b, n, k = w.shape
    m = x.shape[0]
    for name, t in (("x", x), ("out", out)):
        if not t.is_cuda or t.dim() != 2 or t.stride(1) != 1:
            raise ValueError(f"GROUPED_PROJ {name}: a CUDA matrix with dense rows is needed")
    if (x.shape[1] != k or tuple(out.shape) != (m, n // 2 if act in GATED else n) or x.dtype != w.dtype or row_offsets.dtype != torch.int32
            or row_offsets.shape[0] != b + 1):
        raise ValueError(f"GROUPED_PROJ: x {tuple(x.shape)} {x.dtype}, w {tuple(w.shape)} {w.dtype}, out {tuple(out.shape)} do not fit")
    p = N.DenseProblem(x=_ptr(x), w=_ptr(w), y=_ptr(out), ld_x=x.stride(0), ld_y=out.stride(0), batch_w=n * k, k=k, n=n, batch=b, act=act,
                       y_dtype=_dt(out), row_offsets=_ptr(row_offsets))
    p.rows, p.like = m, x
    return p


def interleave_gate(gate, up):
    """Gate and up projections [..., F, K] as a gated `dense` takes them: blocks of 16 rows of each in turn, F padded to a multiple of
    16 with zeros (whose outputs are zero)."""
    f, k = gate.shape[-2:]
    pad = -f % 16
    if pad:
        gate, up = (torch.nn.functional.pad(t, (0, 0, 0, pad)) for t in (gate, up))
    lead = gate.shape[:-2]
    both = torch.stack([gate.reshape(*lead, -1, 16, k), up.reshape(*lead, -1, 16, k)], dim=-3)
    return both.reshape(*lead, 2 * (f + pad), k).contiguous()


def dense_gemm(*problems, weights_const=False) -> None:
    """Runs one or two `dense` problems of the same type (a `grouped_dense` one last)."""
    like, m = problems[0].like, problems[0].rows
    if any(p.like.dtype != like.dtype for p in problems):
        raise ValueError("DENSE_PROJ: the problems of one call have the same type")
    N.check(N.lib().tlaloc_b200_dense_gemm((N.DenseProblem * len(problems))(*problems), len(problems), _dt(like), m,
                                           N.GEMM_WEIGHTS_CONST if weights_const else 0, _stream(like)))


def rmsnorm_pair(x, gain_a, out_a, eps, gain_b=None, out_b=None) -> None:
    """out_a = x / sqrt(mean(x^2) + eps) * gain_a and, if given, the same with gain_b into out_b; x f32 [rows, n]."""
    _dev(x, gain_a, gain_b)
    rows, n = x.shape
    _out("RMSNORM_PAIR out", out_a, (rows, n), (torch.float32, torch.bfloat16), x)
    _out("RMSNORM_PAIR second out", out_b, (rows, n), out_a.dtype, x)
    N.check(N.lib().tlaloc_b200_rmsnorm_pair(_ptr(x), _ptr(gain_a), _ptr(out_a), _ptr(gain_b), _ptr(out_b), _dt(out_a), rows, n, float(eps),
                                             _stream(x)))


def latent_kv_write(low, q_gain, kv_gain, eps, positions, cos, sin, slots, cq, pool, *, q_rank, kv_rank, rot_dim, rot_dims) -> None:
    """low f32 [T, q_rank + kv_rank + rot_dim] -> cq [T, q_rank] (normed) and pool rows [kv_rank | rot_dim] (normed, rotated)."""
    _dev(q_gain, kv_gain, positions, cos, sin, slots, cq, pool)
    T = low.shape[0]
    if low.dtype != torch.float32 or low.stride(1) != 1 or low.shape[1] != q_rank + kv_rank + rot_dim:
        raise ValueError("LATENT_KV_WRITE: low is f32 [T, q_rank + kv_rank + rot_dim] with dense rows")
    if pool.dim() != 3 or positions.shape[0] < T or slots.shape[0] < T or tuple(cos.shape) != (cos.shape[0], rot_dims // 2) or cos.shape != sin.shape:
        raise ValueError("LATENT_KV_WRITE: pool [P, block, row], positions and slots [T], cos and sin [positions, rot_dims / 2]")
    if q_rank:
        _out("LATENT_KV_WRITE cq", cq, (T, q_rank), pool.dtype, low)
    N.check(N.lib().tlaloc_b200_latent_kv_write(
        _ptr(low), low.stride(0), _ptr(q_gain), _ptr(kv_gain), float(eps), _ptr(positions), _ptr(cos), _ptr(sin), _ptr(slots), _ptr(cq),
        _ptr(pool), _dt(pool), pool.shape[2], T, q_rank, kv_rank, rot_dim, rot_dims, pool.shape[0] * pool.shape[1], cos.shape[0], _stream(low)))


def rope_interleaved(x, out, positions, cos, sin, *, rot_dims) -> None:
    """x, out [T, H, width] (strided views of the same type; may be the same): the first rot_dims elements rotated in pairs."""
    T, H, width = x.shape
    if x.shape != out.shape or x.dtype != out.dtype or x.stride(2) != 1 or out.stride(2) != 1 or not (x.is_cuda and out.is_cuda):
        raise ValueError("ROPE_INTERLEAVED: x and out are CUDA tensors [T, H, width] of one type with dense rows")
    _dev(positions, cos, sin)
    N.check(N.lib().tlaloc_b200_rope_interleaved(_ptr(x), x.stride(0), x.stride(1), _ptr(out), out.stride(0), out.stride(1), _dt(x),
                                                 _ptr(positions), _ptr(cos), _ptr(sin), T, H, width, rot_dims, cos.shape[0], _stream(x)))


def latent_attention_scratch_bytes(rows, heads, kv_rank, rot_dim, max_live) -> int:
    return int(N.lib().tlaloc_b200_latent_attention_scratch_bytes(rows, heads, kv_rank, rot_dim, max_live))


def latent_attention(query, pool, block_tables, seq_lens, out, *, kv_rank, scale, window=0, row_tables=None, scratch=None, max_live=0) -> None:
    """query [T, H, kv_rank + rot_dim] over pool [P, block, row] -> out [T, H, kv_rank]; see include/tlaloc_b200.h.
    max_live: a bound on the live positions of any row (0: what the tables and the window allow)."""
    _dev(query, pool, block_tables, seq_lens, out, row_tables, scratch)
    T, H, row = query.shape
    if query.dtype != pool.dtype or pool.dim() != 3:
        raise ValueError("LATENT_ATTENTION: query and pool have one type; pool is [P, block, row]")
    if any(t is not None and t.dtype != torch.int32 for t in (block_tables, seq_lens, row_tables)):
        raise TypeError("LATENT_ATTENTION: tables and lengths are int32")
    if seq_lens.shape[0] < T or (row_tables is not None and row_tables.shape[0] < T):
        raise ValueError("LATENT_ATTENTION: one length and one table per row")
    _out("LATENT_ATTENTION out", out, (T, H, kv_rank), query.dtype, query)
    P, bs, ld = pool.shape
    N.check(N.lib().tlaloc_b200_latent_attention(
        _ptr(query), _ptr(pool), ld, _dt(query), _ptr(block_tables), _ptr(row_tables), _ptr(seq_lens), _ptr(out), _ptr(scratch),
        0 if scratch is None else scratch.numel() * scratch.element_size(), T, H, kv_rank, row - kv_rank, P, bs, block_tables.shape[1],
        block_tables.shape[0], int(window), int(max_live), float(scale), _stream(query)))


def latent_gather(pool, table, out, *, first, keep=0) -> None:
    """out [count, row] = the pool rows of positions 0 .. keep - 1 and first .. of the sequence whose block table is `table` [max_blocks]."""
    _dev(pool, table, out)
    if table.dtype != torch.int32 or table.dim() != 1 or pool.dim() != 3 or out.dtype != pool.dtype:
        raise ValueError("LATENT_GATHER: pool [P, block, row], table i32 [max_blocks], out [count, row] of the pool's type")
    P, bs, ld = pool.shape
    N.check(N.lib().tlaloc_b200_latent_gather(_ptr(pool), ld, _dt(pool), _ptr(table), _ptr(out), out.shape[1], int(first), int(keep), out.shape[0],
                                              out.shape[1], P, bs, table.shape[0], _stream(pool)))


def window_attention_applies(dim, rot_dim, vdim) -> bool:
    return bool(N.lib().tlaloc_b200_window_attention_applies(dim, rot_dim, vdim))


def window_attention(q, k, k_rot, v, out, *, first_query, scale, window=0, keep_first=0, maps=1) -> None:
    """q bf16 [T, H, dim + rot] (contiguous, rotated) over k [L, groups * maps, dim], k_rot [L, rot] (or None) and v [L, groups, vdim]
    (strided views) -> out [T, H * vdim] (a strided view); query i is key first_query + i.  See include/tlaloc_b200.h."""
    _dev(q)
    T, H, qd = q.shape
    L, kh, dim = k.shape
    vh, vdim = v.shape[1:]
    rot = qd - dim
    k_rot = k_rot if rot else None
    if any(t is not None and (t.dtype != torch.bfloat16 or not t.is_cuda or t.stride(-1) != 1) for t in (q, k, k_rot, v)):
        raise ValueError("WINDOW_ATTENTION: bf16 CUDA tensors with dense rows")
    if not out.is_cuda or out.stride(-1) != 1 or out.dtype not in (torch.float32, torch.bfloat16):
        raise ValueError("WINDOW_ATTENTION: out is an f32 or bf16 CUDA matrix with dense rows")
    if (kh != vh * maps or H % kh or v.shape[0] != L or rot < 0 or (rot and tuple(k_rot.shape) != (L, rot))
            or tuple(out.shape) != (T, H * vdim) or v.stride(0) != k.stride(0)):
        raise ValueError(f"WINDOW_ATTENTION: q {tuple(q.shape)}, k {tuple(k.shape)}, v {tuple(v.shape)}, out {tuple(out.shape)} do not fit")
    N.check(N.lib().tlaloc_b200_window_attention(_ptr(q), _ptr(k), k.stride(1), _ptr(k_rot), k_rot.stride(0) if rot else 8, _ptr(v), v.stride(1), k.stride(0),
                                                 _ptr(out), out.stride(0), _dt(out), T, L, int(first_query), H, vh, int(maps), dim, rot, vdim, int(window),
                                                 int(keep_first), float(scale), _stream(q)))


# ---------------------------------------------------------------------- norms on both sides, grouped attention, retention, experts


def residual_norm(y, x, gain_post, eps, *, gain_next=None, out=None, gate=None, parts=None, part_rows=None, part_weights=None) -> None:
    """x += rms_norm(branch) * gain_post with branch = sigmoid(gate) * y + the weighted expert outputs; out = rms_norm(x) * gain_next.
    y f32 [rows, n] or None; gate f32 [rows] (strided); parts [rows * top, n], part_rows i32 and part_weights f32 [rows, top]."""
    _dev(x, gain_post, gain_next, y, parts, part_rows, part_weights)
    rows, n = x.shape
    if (y is not None and (tuple(y.shape) != (rows, n) or y.dtype != torch.float32)) or (gate is not None and gate.shape[0] != rows):
        raise ValueError("RESIDUAL_NORM: y is f32 [rows, n], gate f32 [rows]")
    if out is not None:
        _out("RESIDUAL_NORM out", out, (rows, n), (torch.float32, torch.bfloat16), x)
    kind = _dt(parts if parts is not None else out if out is not None else x)
    if parts is not None and (out is not None and out.dtype != parts.dtype or parts.shape[-1] != n or tuple(part_rows.shape) != tuple(part_weights.shape)
                              or part_rows.dtype != torch.int32):
        raise ValueError("RESIDUAL_NORM: parts [.., n] of the result's type, part_rows i32 and part_weights [rows, top]")
    N.check(N.lib().tlaloc_b200_residual_norm(_ptr(y), _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(parts), _ptr(part_rows),
                                              _ptr(part_weights), part_rows.shape[1] if parts is not None else 0, _ptr(x), _ptr(gain_post),
                                              _ptr(gain_next), _ptr(out), kind, rows, n, float(eps), _stream(x)))


def rotate_part(out, first, heads, dim, *, padded=None, row_ld, head_ld=None, rotate=True, scale=1.0, by_slot=False) -> N.RotatePart:
    """Where one part of a projected row goes (`rotate_rows`): out is the address's tensor, its rows row_ld apart."""
    padded = dim if padded is None else padded
    p = N.RotatePart(out=_ptr(out), out_ld=row_ld, out_head_ld=padded if head_ld is None else head_ld, first=first, heads=heads, dim=dim,
                     padded=padded, rotate=int(rotate), by_slot=int(by_slot), scale=scale)
    p.like = out
    return p


def rotate_rows(rows, parts, positions, cos, sin, *, rot_dims, slots=None, num_slots=0) -> None:
    """rows f32 [T, ld] (dense rows): each part rotated, scaled, narrowed and written to its place."""
    _dev(positions, cos, sin, slots)
    T = rows.shape[0]
    if rows.dtype != torch.float32 or not rows.is_cuda or rows.stride(1) != 1 or positions.shape[0] < T or (slots is not None and slots.shape[0] < T):
        raise ValueError("ROTATE_ROWS: rows f32 [T, ld], positions and slots [T]")
    if any(p.like.dtype != parts[0].like.dtype for p in parts) or tuple(cos.shape) != (cos.shape[0], rot_dims // 2) or cos.shape != sin.shape:
        raise ValueError("ROTATE_ROWS: outputs of one type; cos and sin [positions, rot_dims / 2]")
    N.check(N.lib().tlaloc_b200_rotate_rows(_ptr(rows), rows.stride(0), (N.RotatePart * len(parts))(*parts), len(parts), _dt(parts[0].like),
                                            _ptr(positions), _ptr(cos), _ptr(sin), _ptr(slots), T, rot_dims, num_slots, max(cos.shape[0], 1), _stream(rows)))


def grouped_attention_slices(rows, heads, v_heads, maps, dim, vdim, block_size, dtype, max_live) -> int:
    return int(N.lib().tlaloc_b200_grouped_attention_slices(rows, heads, v_heads, maps, dim, vdim, block_size, _DT[dtype], max_live))


def grouped_attention(q, pool, block_tables, seq_lens, records, *, v_heads, maps, vdim, v_first, scale, slices, window=0, keep_first=0,
                      row_tables=None) -> None:
    """q [T, H, dim] over pool [P, block, row] of rows [v_heads * maps * dim keys | .. | v_heads * vdim values from v_first] -> records f32
    of at least slices * T * H * (vdim + 2) values; see include/tlaloc_b200.h."""
    _dev(q, pool, block_tables, seq_lens, records, row_tables)
    T, H, dim = q.shape
    P, bs, ld = pool.shape
    if q.dtype != pool.dtype or records.dtype != torch.float32 or records.numel() < slices * T * H * (vdim + 2):
        raise ValueError("GROUPED_ATTENTION: q and pool have one type; records are f32 [slices, T, H, vdim + 2]")
    if any(t is not None and t.dtype != torch.int32 for t in (block_tables, seq_lens, row_tables)):
        raise TypeError("GROUPED_ATTENTION: tables and lengths are int32")
    if seq_lens.shape[0] < T or (row_tables is not None and row_tables.shape[0] < T):
        raise ValueError("GROUPED_ATTENTION: one length and one table per row")
    N.check(N.lib().tlaloc_b200_grouped_attention(_ptr(q), _ptr(pool), ld, _dt(q), _ptr(block_tables), _ptr(row_tables), _ptr(seq_lens), _ptr(records),
                                                  slices, T, H, v_heads, maps, dim, vdim, v_first, P, bs, block_tables.shape[1], block_tables.shape[0],
                                                  int(window), int(keep_first), float(scale), _stream(q)))


def map_difference(maps, out, *, rows, heads, vdim, in_ld, lam, keep, eps, slices=0, gate=None) -> None:
    """The difference of two attention maps, normed and gated: maps f32 (records of `slices` slices, or the maps' outputs), gate f32
    [rows, heads] (strided), out [rows, heads * vdim] (strided)."""
    _dev(maps)
    need = max(slices, 1) * rows * heads * 2 * (in_ld + 2 if slices else in_ld)
    if maps.dtype != torch.float32 or maps.numel() < need or tuple(out.shape) != (rows, heads * vdim) or out.stride(1) != 1 or not out.is_cuda:
        raise ValueError("MAP_DIFFERENCE: maps f32 of every head, out [rows, heads * vdim]")
    N.check(N.lib().tlaloc_b200_map_difference(_ptr(maps), slices, _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(out), out.stride(0), _dt(out),
                                               rows, heads, vdim, in_ld, float(lam), float(keep), float(eps), _stream(maps)))


def head_norm_gate(o, gate, out, eps) -> None:
    """o f32 [rows, heads, vdim], gate f32 [rows, heads * vdim] (strided) -> out = o / rms(o) * silu(gate), [rows, heads * vdim]."""
    _dev(o)
    rows, heads, vdim = o.shape
    if o.dtype != torch.float32 or gate.dtype != torch.float32 or gate.stride(1) != 1 or tuple(out.shape) != (rows, heads * vdim) or out.stride(1) != 1:
        raise ValueError("HEAD_NORM_GATE: o and gate f32, out [rows, heads * vdim]")
    N.check(N.lib().tlaloc_b200_head_norm_gate(_ptr(o), _ptr(gate), gate.stride(0), _ptr(out), out.stride(0), _dt(out), rows, heads, vdim, float(eps), _stream(o)))


def _state_shape(state, heads, dim, vdim):
    if state.dtype != torch.float32 or tuple(state.shape[1:]) != (heads, dim, -(-vdim // 4) * 4):
        raise ValueError(f"RETENTION: state {tuple(state.shape)} is not f32 [slots, {heads}, {dim}, vdim rounded up to 4]")


def retention_step(rows, positions, cos, sin, decay, row_states, state, out, *, heads, dim, vdim, rot_dims, k_scale, eps) -> None:
    """One token per row: rows f32 [T, heads * (2 dim + 2 vdim)] = [q | k | v | gate] -> out [T, heads * vdim] and the new states."""
    _dev(positions, cos, sin, decay, row_states, state)
    T = rows.shape[0]
    _state_shape(state, heads, dim, vdim)
    if rows.dtype != torch.float32 or rows.stride(1) != 1 or tuple(out.shape) != (T, heads * vdim) or out.stride(1) != 1 or decay.numel() != heads:
        raise ValueError("RETENTION_STEP: rows f32 [T, ..], out [T, heads * vdim], decay f32 [heads]")
    N.check(N.lib().tlaloc_b200_retention_step(_ptr(rows), rows.stride(0), _ptr(positions), _ptr(cos), _ptr(sin), _ptr(decay), _ptr(row_states), _ptr(state),
                                               _ptr(out), out.stride(0), _dt(out), T, heads, dim, vdim, rot_dims, state.shape[0], max(cos.shape[0], 1),
                                               float(k_scale), float(eps), _stream(state)))


def retention_scan(q, k, v, positions, decay, row_states, state, o) -> None:
    """The tokens of one sequence in order: q, k [T, heads, dim] and v [T, heads, vdim] (heads side by side, each padded to a row of its
    own length) -> o f32 [T, heads, vdim] and the new state."""
    T, heads, vdim = o.shape
    _dev(decay, state, o)
    dim = state.shape[2]
    _state_shape(state, heads, dim, vdim)
    for t in (q, k, v):
        if not t.is_cuda or not t.is_contiguous() or t.shape[:2] != (T, heads) or t.dtype != q.dtype:
            raise ValueError("RETENTION_SCAN: q, k, v are contiguous [T, heads, ..] of one type")
    N.check(N.lib().tlaloc_b200_retention_scan(_ptr(q), _ptr(k), q.shape[2], _ptr(v), v.shape[2], _dt(q), _ptr(positions), _ptr(decay), _ptr(row_states),
                                               _ptr(state), _ptr(o), T, heads, dim, vdim, state.shape[0], _stream(state)))


def retention_chunks_scratch_bytes(tokens, heads, dim, vdim) -> int:
    return int(N.lib().tlaloc_b200_retention_chunks_scratch_bytes(tokens, heads, dim, vdim))


def retention_chunks_applies(dim, vdim) -> bool:
    return bool(N.lib().tlaloc_b200_retention_chunks_applies(dim, vdim))


def retention_chunks(q, k, v, positions, decay, row_states, state, o, scratch=None) -> None:
    """`retention_scan` on the tensor cores, bf16: what pads the rows of q, k and v must be zero; scratch f32 of
    retention_chunks_scratch_bytes."""
    T, heads, vdim = o.shape
    _dev(decay, state, o, scratch)
    dim = state.shape[2]
    _state_shape(state, heads, dim, vdim)
    for t in (q, k, v):
        if not t.is_cuda or not t.is_contiguous() or t.shape[:2] != (T, heads) or t.dtype != torch.bfloat16:
            raise ValueError("RETENTION_CHUNKS: q, k, v are contiguous bf16 [T, heads, ..]")
    N.check(N.lib().tlaloc_b200_retention_chunks(_ptr(q), _ptr(k), q.shape[2], _ptr(v), v.shape[2], _ptr(positions), _ptr(decay), _ptr(row_states),
                                                 _ptr(state), _ptr(o), _ptr(scratch), 0 if scratch is None else scratch.numel() * scratch.element_size(),
                                                 T, heads, dim, vdim, state.shape[0], _stream(state)))


def moe_route(logits, ids, weights, offsets, entry_rows, row_tokens, *, experts) -> None:
    """logits f32 [T, >= experts] (strided) -> the chosen experts and their weights [T, top], and the entries sorted by expert."""
    _dev(ids, weights, offsets, entry_rows, row_tokens)
    T, top = ids.shape
    if logits.dtype != torch.float32 or logits.stride(1) != 1 or logits.shape[0] != T or offsets.shape[0] != experts + 1:
        raise ValueError("MOE_ROUTE: logits f32 [T, ..], offsets [experts + 1]")
    N.check(N.lib().tlaloc_b200_moe_route(_ptr(logits), logits.stride(0), _ptr(ids), _ptr(weights), _ptr(offsets), _ptr(entry_rows), _ptr(row_tokens), T,
                                          experts, top, _stream(ids)))


def gather_rows(x, rows, out) -> None:
    """out[r] = x[rows[r]]."""
    _dev(x, rows, out)
    if rows.dtype != torch.int32 or out.dtype != x.dtype or out.shape != (rows.shape[0], x.shape[1]):
        raise ValueError("GATHER_ROWS: rows i32 [count], out [count, n] of x's type")
    N.check(N.lib().tlaloc_b200_gather_rows(_ptr(x), _ptr(rows), _ptr(out), rows.shape[0], x.shape[1] * x.element_size(), _stream(x)))
