"""The operators of a latent-attention layer through the C ABI, each against its equation in f64 (needs a B200).

Attention inputs are made so that a mistake shows: besides random ones, a single key is aligned with the query ("needle") at a
chosen distance, so that seeing it or not changes the whole output."""
import math

import pytest
import torch

import latent_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(autouse=True)
def no_wait_runs_out():
    """Every device-side wait is bounded; one that runs out leaves a status word (and a wrong result)."""
    yield
    from tlaloc_b200 import _native

    torch.cuda.synchronize()
    assert _native.lib().tlaloc_b200_device_status() == 0


def gen(seed):
    g = torch.Generator(device=DEV)
    g.manual_seed(seed)
    return g


def randn(*shape, seed=0, dtype=torch.float32):
    return torch.randn(shape, device=DEV, generator=gen(seed)).to(dtype)


def tol(dtype, k=1.0):
    return (2e-5 if dtype == torch.float32 else 1.2e-2) * k


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,n", [(1, 8), (3, 72), (5, 257), (2, 4096), (2, 10000)])
def test_pair_of_norms(dtype, rows, n):
    from tlaloc_b200 import ops

    x, ga, gb = 3 * randn(rows, n), randn(n, seed=1), randn(n, seed=2)
    a, b = torch.empty((rows, n), device=DEV, dtype=dtype), torch.empty((rows, n), device=DEV, dtype=dtype)
    ops.rmsnorm_pair(x, ga, a, 1e-3, gb, b)
    want = oracle.rms(x.double(), 1e-3)
    assert float((a.double() - want * ga.double()).abs().max()) <= tol(dtype, 4)
    assert float((b.double() - want * gb.double()).abs().max()) <= tol(dtype, 4)
    single = torch.empty_like(a)
    ops.rmsnorm_pair(x, ga, single, 1e-3)
    assert torch.equal(single, a)
    tiny = torch.full((1, n), 1e-4, device=DEV)  # eps decides
    ops.rmsnorm_pair(tiny, torch.ones(n, device=DEV), a[:1], 1e-3)
    assert abs(float(a[0, 0]) - 1e-4 / math.sqrt(1e-8 + 1e-3)) <= 1e-2 * 3e-3


ROTATIONS = [dict(dims=8, base=100.0), dict(dims=16, base=10000.0, scaling=dict(factor=4.0, original=128, fast=8.0, slow=1.0)),
             dict(dims=2, base=10.0, scaling=dict(factor=2.0, original=64, fast=32.0, slow=16.0)),
             dict(dims=64, base=1e6, scaling=dict(factor=40.0, original=4096, fast=32.0, slow=1.0))]


def tables(rot, n):
    from tlaloc_b200.rotary import Rotation, YarnScaling, pair_tables

    s = rot.get("scaling")
    r = Rotation(rot["dims"], rot["base"], YarnScaling(s["factor"], s["original"], s["fast"], s["slow"]) if s else None)
    return tuple(torch.from_numpy(t).to(DEV) for t in pair_tables(r, n))


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rot", ROTATIONS)
@pytest.mark.parametrize("extra", [0, 5])
def test_interleaved_rotation(dtype, rot, extra):
    """Strided input and output, in place too; dimensions past the rotated ones are copied."""
    from tlaloc_b200 import ops

    cos, sin = tables(rot, 3000)
    pos = torch.tensor([0, 1, 2, 63, 64, 511, 2999], dtype=torch.int32, device=DEV)
    width = rot["dims"] + extra
    x = randn(7, 3, width + 4, dtype=dtype)
    out = torch.full((7, 3, width + 9), 5.0, device=DEV, dtype=dtype)
    ops.rope_interleaved(x[:, :, 4:], out[:, :, 6:6 + width], pos, cos, sin, rot_dims=rot["dims"])
    want = oracle.rotate(x[:, :, 4:].double().cpu(), pos.cpu(), rot).to(DEV)
    assert float((out[:, :, 6:6 + width].double() - want).abs().max()) <= tol(dtype, 6)
    assert bool((out[:, :, :6] == 5).all()) and bool((out[:, :, 6 + width:] == 5).all())
    ops.rope_interleaved(x[:, :, 4:], x[:, :, 4:], pos, cos, sin, rot_dims=rot["dims"])
    assert torch.equal(x[:, :, 4:], out[:, :, 6:6 + width])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot_dim,rot_dims", [(56, 48, 8, 8), (300, 512, 64, 64), (24, 40, 20, 16), (0, 72, 8, 8)])
def test_norms_rotation_and_cache_write(dtype, q_rank, kv_rank, rot_dim, rot_dims):
    from tlaloc_b200 import ops

    rot = dict(dims=rot_dims, base=500.0, scaling=dict(factor=4.0, original=64, fast=8.0, slow=1.0))
    cos, sin = tables(rot, 400)
    T, row = 6, kv_rank + rot_dim
    low = 2 * randn(T, q_rank + row + 3)[:, :q_rank + row]
    qg, kg = randn(max(q_rank, 1), seed=1), randn(kv_rank, seed=2)
    pos = torch.tensor([0, 1, 17, 64, 399, 5], dtype=torch.int32, device=DEV)
    slots = torch.tensor([3, 0, 31, 16, 15, -1], dtype=torch.int32, device=DEV)
    pool = torch.full((2, 16, -(-row // 8) * 8), 9.0, device=DEV, dtype=dtype)
    cq = torch.empty((T, q_rank), device=DEV, dtype=dtype)
    ops.latent_kv_write(low, qg, kg, 1e-4, pos, cos, sin, slots, cq, pool, q_rank=q_rank, kv_rank=kv_rank, rot_dim=rot_dim, rot_dims=rot_dims)
    x = low.double().cpu()
    flat = pool.view(32, -1)
    if q_rank:
        want = oracle.rms(x[:, :q_rank], 1e-4) * qg.double().cpu()
        assert float((cq.double().cpu() - want).abs().max()) <= tol(dtype, 6)
    latent = oracle.rms(x[:, q_rank:q_rank + kv_rank], 1e-4) * kg.double().cpu()
    shared = oracle.rotate(x[:, q_rank + kv_rank:], pos.cpu(), rot)
    want = torch.cat([latent, shared], 1)[:5]
    got = flat[slots[:5].long()][:, :row].double().cpu()
    assert float((got - want).abs().max()) <= tol(dtype, 12)
    untouched = [i for i in range(32) if i not in slots.tolist()]
    assert bool((flat[untouched] == 9).all())


# ---------------------------------------------------------------------------------------------- absorbed attention

def paged(rows_by_seq, block, row, dtype, seed=0):
    """Rows of several sequences scattered over pages that held something else before; block tables of unequal length."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-r.shape[0] // block) for r in rows_by_seq]
    pages = 1 + torch.randperm(sum(need) + 3, generator=g)
    pool = 50 * randn(sum(need) + 4, block, -(-row // 8) * 8, seed=seed, dtype=dtype)  # whatever a freed page still holds
    table = torch.zeros((len(need), max(need)), dtype=torch.int32)
    at = 0
    for s, (r, n) in enumerate(zip(rows_by_seq, need)):
        table[s, :n] = pages[at:at + n].int()
        flat = torch.cat([r, pool[0, :1, :row].repeat(n * block - r.shape[0], 1).to(r)]) if n * block > r.shape[0] else r
        for i in range(n):
            keep = min(block, r.shape[0] - i * block)
            pool[pages[at + i], :keep, :row] = flat[i * block:i * block + keep]
        at += n
    return pool, table.to(DEV)


def attend(q, rows, kv_rank, scale, lo, hi):
    k = rows[lo:hi].double()
    return torch.softmax(q.double() @ k.T * scale, -1) @ k[:, :kv_rank]


SHAPES = [(3, 48, 8), (16, 256, 32), (17, 128, 64), (40, 512, 64), (5, 36, 6)]  # heads, kv_rank, rot_dim


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,kv_rank,rot_dim", SHAPES)
@pytest.mark.parametrize("window", [0, 1, 64, 65, 200])
@pytest.mark.parametrize("block", [16, 64])
def test_absorbed_attention_over_pages(dtype, heads, kv_rank, rot_dim, window, block):
    """Unequal rows (lengths at and around tile, page and window edges) against each alone; several rows of one sequence."""
    from tlaloc_b200 import ops

    row = kv_rank + rot_dim
    lens = [1, 2, 63, 64, 65, 200, 201, 333]
    seqs = [randn(n, row, seed=n, dtype=dtype) for n in lens]
    pool, table = paged(seqs, block, row, dtype)
    which = torch.tensor([0, 1, 2, 3, 4, 5, 6, 7, 7, 7], dtype=torch.int32, device=DEV)
    ends = torch.tensor(lens + [100, 332], dtype=torch.int32, device=DEV)
    q = randn(len(which), heads, row, seed=9, dtype=dtype)
    scale = 1.7 * row ** -0.5
    out = torch.empty((len(which), heads, kv_rank), device=DEV, dtype=dtype)
    results = []
    for scratch in (None, torch.empty((1 << 22,), device=DEV)):
        ops.latent_attention(q, pool, table, ends, out, kv_rank=kv_rank, scale=scale, window=window, row_tables=which, scratch=scratch)
        results.append(out.clone())
    for t in range(len(which)):
        hi = int(ends[t])
        want = attend(q[t], seqs[int(which[t])], kv_rank, scale, max(0, hi - window) if window else 0, hi)
        for r in results:
            assert float((r[t].double() - want).abs().max()) <= tol(dtype, 2.5), (t, hi)
    one = torch.empty((1, heads, kv_rank), device=DEV, dtype=dtype)
    ops.latent_attention(q[7:8], pool, table, ends[7:8], one, kv_rank=kv_rank, scale=scale, window=window, row_tables=which[7:8])
    assert float((one[0].double() - results[0][7].double()).abs().max()) <= tol(dtype)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("window", [40, 64, 129, 700])
def test_absorbed_attention_needle_at_the_window_edge(dtype, window):
    """One key matches the query and carries its own value: just inside the window it is the output, just outside it is not there."""
    from tlaloc_b200 import ops

    heads, kv_rank, rot_dim, end = 20, 64, 16, 1000
    row = kv_rank + rot_dim
    for distance in (0, 1, window - 2, window - 1, window, window + 1):
        rows = 0.1 * randn(end, row, seed=distance, dtype=dtype)
        q = randn(1, heads, row, seed=3, dtype=dtype)
        at = end - 1 - distance
        rows[at] = (8 * q[0, 0]).to(dtype)  # head 0's needle
        pool, table = paged([rows], 64, row, dtype)
        out = torch.empty((1, heads, kv_rank), device=DEV, dtype=dtype)
        ops.latent_attention(q, pool, table, torch.tensor([end], dtype=torch.int32, device=DEV), out, kv_rank=kv_rank, scale=0.1, window=window,
                             scratch=torch.empty((1 << 20,), device=DEV))
        needle = rows[at, :kv_rank].double()
        share = float((out[0, 0].double() @ needle) / (needle @ needle))
        assert share > 0.99 if distance < window else abs(share) < 0.1, (distance, share)
        want = attend(q[0], rows, kv_rank, 0.1, max(0, end - window), end)
        assert float((out[0].double() - want).abs().max()) <= tol(dtype, 12)


# ---------------------------------------------------------------------------------------------- expanded attention

def window_reference(q, k, k_rot, v, first, scale, window):
    T, H, L = q.shape[0], q.shape[1], k.shape[0]
    kk = torch.cat([k, k_rot[:, None].expand(L, H, k_rot.shape[1])], -1).double()
    d = (first + torch.arange(T, device=DEV))[:, None] - torch.arange(L, device=DEV)[None, :]
    seen = (d >= 0) & (d < window) if window else d >= 0
    s = (torch.einsum("ihd,jhd->hij", q.double(), kk) * scale).masked_fill(~seen, -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v.double()).reshape(T, -1)


@pytest.mark.parametrize("heads,dim,rot,vdim", [(3, 24, 8, 40), (2, 128, 64, 128), (2, 64, 32, 64), (1, 72, 16, 136), (2, 192, 64, 256), (2, 64, 0, 96)])
@pytest.mark.parametrize("T,first,window", [(1, 0, 0), (2, 5, 3), (128, 0, 0), (129, 0, 1), (100, 28, 128), (300, 400, 129), (260, 127, 50), (130, 1000, 0)])
def test_expanded_attention(heads, dim, rot, vdim, T, first, window):
    from tlaloc_b200 import ops

    L = first + T
    q = 2 * randn(T, heads, dim + rot, seed=1)
    q = q.to(torch.bfloat16)
    kv = randn(L, heads, dim + vdim, seed=2, dtype=torch.bfloat16)
    lat = randn(L, 16 + rot, seed=3, dtype=torch.bfloat16)
    out = torch.full((T, heads * vdim + 16), 5.0, device=DEV, dtype=torch.bfloat16)
    scale = (dim + rot) ** -0.5
    ops.window_attention(q, kv[:, :, :dim], lat[:, 16:], kv[:, :, dim:], out[:, :heads * vdim], first_query=first, scale=scale, window=window)
    want = window_reference(q, kv[:, :, :dim], lat[:, 16:], kv[:, :, dim:], first, scale, window)
    assert float((out[:, :heads * vdim].double() - want).abs().max()) <= 2.5e-2
    assert bool((out[:, heads * vdim:] == 5).all())


@pytest.mark.parametrize("window", [64, 127, 128, 129, 300])
def test_expanded_attention_needle_at_the_window_edge(window):
    """As above, for queries at several places of a portion; growing needles also force the running maximum up late."""
    from tlaloc_b200 import ops

    heads, dim, rot, vdim, T, first = 2, 48, 16, 64, 200, 350
    for i in (0, 1, 127, 128, 199):
        for distance in (0, window - 1, window):
            q = randn(T, heads, dim + rot, seed=1, dtype=torch.bfloat16)
            kv = 0.1 * randn(first + T, heads, dim + vdim, seed=2, dtype=torch.bfloat16)
            k_rot = 0.1 * randn(first + T, rot, seed=3, dtype=torch.bfloat16)
            at = first + i - distance
            kv[at, 0, :dim] = 8 * q[i, 0, :dim]
            kv[at, 0, dim:] = 3.0
            out = torch.empty((T, heads * vdim), device=DEV, dtype=torch.bfloat16)
            ops.window_attention(q, kv[:, :, :dim], k_rot, kv[:, :, dim:], out, first_query=first, scale=0.2, window=window)
            got = float(out[i, :vdim].float().mean())
            assert abs(got - 3.0) < 0.05 if distance < window else abs(got) < 0.2, (i, distance, got)
            want = window_reference(q, kv[:, :, :dim], k_rot, kv[:, :, dim:], first, 0.2, window)
            assert float((out.double() - want).abs().max()) <= 2e-2


def test_the_same_launches_many_times_over():
    """A whole GPU of CTAs whose loads contend: every repetition gives the same bits, prompt portions and decoding alike."""
    from tlaloc_b200 import ops

    T, L, heads = 1024, 3072, 32
    q, kv, lat = randn(T, heads, 192, dtype=torch.bfloat16), randn(L, heads, 256, seed=1, dtype=torch.bfloat16), randn(L, 64, seed=2, dtype=torch.bfloat16)
    first = None
    for _ in range(150):
        out = torch.empty((T, heads * 128), device=DEV, dtype=torch.bfloat16)
        ops.window_attention(q, kv[:, :, :128], lat, kv[:, :, 128:], out, first_query=L - T, scale=0.07, window=2048)
        first = out if first is None else first
        assert torch.equal(out, first)
    pool = randn(48 * 33 + 1, 64, 576, dtype=torch.bfloat16)
    table = (1 + torch.randperm(48 * 33, device=DEV)).int().view(48, 33)
    ends, ql = torch.full((48,), 2100, dtype=torch.int32, device=DEV), randn(48, heads, 576, seed=3, dtype=torch.bfloat16)
    scratch, first = torch.empty((1 << 24,), device=DEV), None
    for _ in range(150):
        out = torch.empty((48, heads, 512), device=DEV, dtype=torch.bfloat16)
        ops.latent_attention(ql, pool, table, ends, out, kv_rank=512, scale=0.04, window=2000, scratch=scratch)
        first = out if first is None else first
        assert torch.equal(out, first)


@pytest.mark.parametrize("dtype", TYPES)
def test_gather_of_a_sequence_from_its_pages(dtype):
    from tlaloc_b200 import ops

    row = 48 + 8
    rows = randn(333, row, dtype=dtype)
    pool, table = paged([randn(70, row, seed=4, dtype=dtype), rows], 64, row, dtype)
    for first, count in ((0, 333), (0, 1), (63, 2), (64, 200), (300, 33)):
        out = torch.empty((count, row), device=DEV, dtype=dtype)
        ops.latent_gather(pool, table[1], out, first=first)
        assert torch.equal(out, rows[first:first + count])


def test_bad_arguments_are_refused():
    from tlaloc_b200 import ops
    from tlaloc_b200._native import KernelError

    pool, table = paged([randn(70, 56)], 64, 56, torch.float32)
    q, out, ends = randn(1, 3, 56), torch.empty((1, 3, 48), device=DEV), torch.tensor([70], dtype=torch.int32, device=DEV)
    with pytest.raises(TypeError):
        ops.latent_attention(q, pool, table.long(), ends, out, kv_rank=48, scale=0.1)
    with pytest.raises(ValueError):
        ops.latent_attention(q.bfloat16(), pool, table, ends, out, kv_rank=48, scale=0.1)
    with pytest.raises(KernelError):
        ops.latent_attention(q, pool[:, :, :40].contiguous(), table, ends, out, kv_rank=48, scale=0.1)
    with pytest.raises(KernelError):
        ops.latent_gather(pool, table[0], torch.empty((200, 56), device=DEV), first=0)
    kv, kr = randn(4, 2, 48, dtype=torch.bfloat16), randn(4, 8, dtype=torch.bfloat16)
    with pytest.raises(KernelError):  # the last query has no key
        ops.window_attention(randn(3, 2, 32, dtype=torch.bfloat16), kv[:, :, :24], kr, kv[:, :, 24:],
                             torch.empty((3, 48), device=DEV, dtype=torch.bfloat16), first_query=2, scale=0.1)
