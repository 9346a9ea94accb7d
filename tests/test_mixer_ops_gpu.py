"""The operators of decoders with mixers of several kinds against plain f64 restatements of their equations (needs a B200)."""
import math

import pytest
import torch

import videdra_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16


@pytest.fixture(autouse=True)
def no_wait_runs_out():
    yield
    from tlaloc_b200 import _native

    torch.cuda.synchronize()
    assert _native.lib().tlaloc_b200_device_status() == 0


def randn(*shape, seed=0, dtype=F32, std=1.0):
    return (std * torch.randn(shape, generator=torch.Generator().manual_seed(seed))).to(dtype).to(DEV)


def near(got, want, tol):
    want = want.double()
    err = float((got.cpu().double() - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), err


# ---------------------------------------------------------------------------------------------- projections

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m,f,k", [(1, 16, 64), (5, 50, 72), (33, 304, 336), (64, 200, 4096), (130, 96, 256), (700, 1000, 512), (3, 8, 20)])
@pytest.mark.parametrize("act", ["silu", "gelu"])
def test_gated_projection(m, f, k, act, dtype):
    from tlaloc_b200 import _native as N
    from tlaloc_b200 import ops

    x, gate, up = randn(m, k, dtype=dtype), randn(f, k, seed=1, dtype=dtype, std=k ** -0.5), randn(f, k, seed=2, dtype=dtype, std=k ** -0.5)
    w = ops.interleave_gate(gate, up)
    fp = w.shape[0] // 2
    assert fp % 16 == 0 and fp >= f
    out = torch.full((m, fp), float("nan"), device=DEV, dtype=dtype)
    ops.dense_gemm(ops.dense(x, w, out, act={"silu": N.ACT_SILU_MUL, "gelu": N.ACT_GELU_TANH_MUL}[act]), weights_const=True)
    xd, g, u = x.cpu().double(), gate.cpu().double(), up.cpu().double()
    want = (oracle.silu if act == "silu" else oracle.gelu_tanh)(xd @ g.T) * (xd @ u.T)
    near(out[:, :f], want, 1e-5 if dtype == F32 else 1e-2)
    assert torch.all(out[:, f:] == 0)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("sizes,n,k", [([3, 0, 17, 1, 0, 40], 64, 48), ([0, 0, 5], 288, 336), ([130, 2, 300, 0, 64, 65], 96, 128), ([1] * 40 + [0] * 9 + [33], 128, 72),
                                       ([513, 700, 5], 256, 256)])
@pytest.mark.parametrize("gated", [False, True])
def test_grouped_projection(sizes, n, k, gated, dtype):
    """Weights with no rows, one, and more than a tile's; alone and behind a projection of other rows in the same call."""
    from tlaloc_b200 import _native as N
    from tlaloc_b200 import ops

    rows, e = sum(sizes), len(sizes)
    offsets = torch.tensor([0] + torch.tensor(sizes).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
    x, w = randn(rows, k, dtype=dtype), randn(e, n, k, seed=1, dtype=dtype, std=k ** -0.5)
    cols = n // 2 if gated else n
    out = torch.full((rows, cols), float("nan"), device=DEV, dtype=dtype)
    act = N.ACT_SILU_MUL if gated else N.ACT_NONE
    grouped = ops.grouped_dense(x, w, out, offsets, act=act)
    h, w2 = randn(7, 64, seed=3, dtype=dtype), randn(40, 64, seed=4, dtype=dtype)
    y2 = torch.full((7, 40), float("nan"), device=DEV)
    for beside in (False, True):
        out.fill_(float("nan"))
        ops.dense_gemm(*([ops.dense(h, w2, y2)] if beside else []), grouped)
        lo = 0
        for i, s in enumerate(sizes):
            if s == 0:
                continue
            z = x[lo:lo + s].cpu().double() @ w[i].cpu().double().T
            if gated:
                z = z.reshape(s, -1, 2, 16)
                z = (oracle.silu(z[:, :, 0]) * z[:, :, 1]).reshape(s, cols)
            near(out[lo:lo + s], z, 1e-5 if dtype == F32 else 1e-2)
            lo += s
    near(y2, h.cpu().double() @ w2.cpu().double().T, 1e-5)


# ---------------------------------------------------------------------------------------------- experts

@pytest.mark.parametrize("tokens,experts,top", [(1, 1, 1), (1, 11, 4), (37, 5, 5), (128, 64, 8), (129, 64, 8), (300, 33, 2), (64, 1000, 31), (2048, 128, 6)])
def test_routing(tokens, experts, top):
    from tlaloc_b200 import ops

    z = randn(tokens, experts + 3, seed=tokens)
    z[tokens // 2, :experts] = 0.25  # equal logits: the first ones
    ids, rows_of = (torch.full((tokens, top), -1, dtype=torch.int32, device=DEV) for _ in range(2))
    weights = torch.zeros((tokens, top), device=DEV)
    offsets, tokens_of = torch.zeros((experts + 1,), dtype=torch.int32, device=DEV), torch.full((tokens * top,), -1, dtype=torch.int32, device=DEV)
    ops.moe_route(z, ids, weights, offsets, rows_of, tokens_of, experts=experts)
    zc = z[:, :experts].cpu().double()
    want = oracle.route(zc, top)
    got = torch.zeros_like(want).scatter_(1, ids.cpu().long(), weights.cpu().double())
    near(got, want, 1e-6)
    assert ids[tokens // 2].tolist() == list(range(top))
    ids, rows_of, off = ids.cpu().long(), rows_of.cpu().long(), offsets.cpu()
    assert off[0] == 0 and off[-1] == tokens * top
    assert torch.equal(torch.diff(off).long(), torch.bincount(ids.flatten(), minlength=experts))
    flat = rows_of.flatten()
    assert torch.equal(flat.sort().values, torch.arange(tokens * top))
    assert torch.all((flat >= off[ids.flatten()]) & (flat < off[ids.flatten() + 1]))
    assert torch.equal(tokens_of.cpu().long()[flat], torch.arange(tokens).repeat_interleave(top))
    for dtype, n in ((BF16, 72), (F32, 5), (BF16, 13)):
        h, out = randn(tokens, n, dtype=dtype), torch.empty((tokens * top, n), device=DEV, dtype=dtype)
        ops.gather_rows(h, tokens_of, out)
        assert torch.equal(out, h[tokens_of.long()])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,n", [(1, 336), (5, 44), (70, 4096), (3, 10000), (2, 7)])
@pytest.mark.parametrize("kind", ["plain", "experts", "experts and shared", "last"])
def test_residual_norm(rows, n, kind, dtype):
    from tlaloc_b200 import ops

    eps, top = 1e-4, 3
    x, y, a, b = randn(rows, n), randn(rows, n, seed=1, std=3.0), randn(n, seed=2), randn(n, seed=3)
    parts, weights, logits = randn(rows * top, n, seed=4, dtype=dtype), randn(rows, top, seed=5), randn(rows, 4, seed=6)
    order = torch.randperm(rows * top, generator=torch.Generator().manual_seed(7)).to(torch.int32).reshape(rows, top).to(DEV)
    d = lambda t: t.cpu().double()
    branch, kw = d(y), {}
    if kind.startswith("experts"):
        kw = dict(parts=parts, part_rows=order, part_weights=weights)
        branch = (d(parts)[order.cpu().long()] * d(weights)[:, :, None]).sum(1)
        if kind.endswith("shared"):
            kw["gate"] = logits[:, 3]
            branch = branch + oracle.sigmoid(d(logits)[:, 3:]) * d(y)
    want_x = d(x) + oracle.rms(branch, eps) * d(a)
    out = None if kind == "last" else torch.empty((rows, n), device=DEV, dtype=dtype)
    ops.residual_norm(None if kind == "experts" else y, x, a, eps, gain_next=b, out=out, **kw)
    near(x, want_x, 1e-5)
    if out is not None:
        near(out, oracle.rms(want_x, eps) * d(b), 1e-5 if dtype == F32 else 8e-3)


# ---------------------------------------------------------------------------------------------- rotation

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim,padded,dims", [(32, 32, 32), (24, 32, 16), (10, 16, 6), (64, 64, 8), (7, 16, 2), (16, 16, 0)])
def test_rotation_into_rows_and_slots(dim, padded, dims, dtype):
    from tlaloc_b200 import ops
    from tlaloc_b200.rotary import Rotation, pair_tables

    T, H, G = 9, 3, 2
    rot = {"base": 500.0, "dims": dims}
    src = randn(T, (H + G) * dim + 4)
    positions = torch.arange(T, dtype=torch.int32, device=DEV)
    cos, sin = (torch.from_numpy(t).to(DEV) for t in pair_tables(Rotation(dims, 500.0), 40))
    q, pool = torch.full((T, H, padded), 9.0, device=DEV, dtype=dtype), torch.full((4, 4, G * padded + 8), 9.0, device=DEV, dtype=dtype)
    slots = torch.tensor([5, 4, -1, 12, 0, 15, 6, 7, 99], dtype=torch.int32, device=DEV)
    ops.rotate_rows(src, [ops.rotate_part(q, 0, H, dim, padded=padded, row_ld=H * padded, scale=0.5),
                          ops.rotate_part(pool, H * dim, G, dim, padded=padded, row_ld=G * padded + 8, by_slot=True)],
                    positions, cos, sin, rot_dims=dims, slots=slots, num_slots=16)
    x = src.cpu().double()[:, :(H + G) * dim].reshape(T, H + G, dim)
    want = oracle.rotate_half(x, rot) if dims else x
    tol = 1e-6 if dtype == F32 else 4e-3
    near(q[:, :, :dim], 0.5 * want[:, :H], tol)
    assert torch.all(q[:, :, dim:] == 0)
    flat = pool.view(16, -1)
    for t, s in enumerate(slots.tolist()):
        if 0 <= s < 16:
            near(flat[s, :G * padded].view(G, padded)[:, :dim], want[t, H:], tol)
    assert torch.all(flat[1:4] == 9.0) and torch.all(flat[8:12] == 9.0) and torch.all(flat[:, G * padded:] == 9.0)


# ---------------------------------------------------------------------------------------------- attention

def paged(T, lens, row, dtype, blocks=40, bs=64, seed=0):
    """A pool of random rows, and per table its pages in any order; the padding page and dead rows hold NaN."""
    g = torch.Generator().manual_seed(seed)
    M = max(-(-l // bs) for l in lens)
    pages = (1 + torch.randperm(blocks - 1, generator=g))[:len(lens) * M].reshape(len(lens), M).to(torch.int32)
    pool = torch.randn((blocks, bs, row), generator=g).to(dtype)
    live = torch.zeros((blocks, bs), dtype=torch.bool)
    for i, l in enumerate(lens):
        for p in range(l):
            live[pages[i, p // bs], p % bs] = True
    pool[~live] = float("nan")
    return pool.to(DEV), pages.to(DEV), M


def seen(n, window, keep):
    return torch.tensor([j for j in range(n) if not window or n - 1 - j < window or j < keep])


def plain(q, k, v, scale):
    """q [dim], k [n, dim], v [n, vdim]"""
    return torch.softmax(k @ q * scale, 0) @ v


ATTENTION = [  # heads per map, groups, maps, dim, vdim
    (6, 2, 2, 32, 48), (8, 1, 2, 64, 128), (20, 2, 2, 16, 16), (4, 4, 1, 128, 64), (40, 2, 1, 64, 256), (2, 2, 2, 128, 256), (12, 4, 2, 48, 80), (3, 1, 2, 24, 40)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,groups,maps,dim,vdim", ATTENTION)
@pytest.mark.parametrize("window,keep", [(0, 0), (100, 0), (64, 3), (33, 70), (1, 0), (500, 8)])
def test_grouped_attention_over_pages(heads, groups, maps, dim, vdim, window, keep, dtype):
    """Lengths around pages, groups and windows; one key outside every window stands out and must not be seen, one just inside and one
    kept key must be."""
    from tlaloc_b200 import ops

    lens = [1, 2, 16, 17, 64, 65, 101, 130]
    T, H, row = len(lens), heads * maps, groups * (maps * dim + vdim) + 8
    v_first = groups * maps * dim + 8
    pool, tables, M = paged(T, lens, row, dtype)
    q, scale = randn(T, H, dim, seed=1, dtype=dtype), dim ** -0.5
    for t, l in enumerate(lens):  # needles: the same key for every head, in the query's direction
        for place in (l - 1 - window, l - window, keep - 1, keep):
            if 0 <= place < l:
                r = pool[tables[t, place // 64], place % 64]
                for g in range(groups):
                    for m in range(maps):
                        r[(g * maps + m) * dim:(g * maps + m + 1) * dim] = 1.5 * q[t, g * (H // groups) + m]
    sl = torch.tensor(lens, dtype=torch.int32, device=DEV)
    order = torch.tensor([3, 0, 5, 1, 7, 2, 6, 4], dtype=torch.int32, device=DEV)
    inverse = torch.argsort(order.long())
    for slices in ({1, 3} if dtype == BF16 and dim % 16 == 0 and vdim % 16 == 0 else {1}):
        records = torch.full((slices, T, H, vdim + 2), float("nan"), device=DEV)
        ops.grouped_attention(q, pool, tables[order.long()].contiguous(), sl, records, v_heads=groups, maps=maps, vdim=vdim, v_first=v_first, scale=scale,
                              slices=slices, window=window, keep_first=keep, row_tables=inverse.to(torch.int32))
        r = records.cpu().double()
        top = r[..., 0].max(0).values
        f = torch.where(torch.isinf(r[..., 0]), torch.zeros(()).double(), torch.exp2(r[..., 0] - top))
        acc = torch.where(f[..., None] > 0, r[..., 2:] * f[..., None], torch.zeros(()).double()).sum(0)
        got = acc / (r[..., 1] * f).sum(0)[..., None]
        for t, l in enumerate(lens):
            j = seen(l, window, keep)
            rows = pool[tables[t, j // 64].long(), (j % 64).to(DEV)].cpu().double()
            for h in range(H):
                g = h // (H // groups)
                kh = g * maps + h % maps
                want = plain(q[t, h].cpu().double(), rows[:, kh * dim:(kh + 1) * dim], rows[:, v_first + g * vdim:v_first + (g + 1) * vdim], scale)
                near(got[t, h], want, 2e-5)


@pytest.mark.parametrize("heads,groups,maps,dim,vdim", [a for a in ATTENTION if a[3] % 16 == 0])
@pytest.mark.parametrize("T,L,window,keep", [(200, 200, 0, 0), (130, 300, 70, 0), (130, 300, 70, 5), (40, 700, 128, 129), (257, 600, 33, 64), (16, 500, 1, 1), (5, 5, 3, 9),
                                             (129, 900, 300, 300)])
def test_grouped_window_attention(heads, groups, maps, dim, vdim, T, L, window, keep):
    from tlaloc_b200 import ops

    H = heads * maps
    q, kv = randn(T, H, dim, seed=2, dtype=BF16), randn(L, groups * (maps * dim + vdim), seed=3, dtype=BF16)
    k, v = kv[:, :groups * maps * dim].view(L, groups * maps, dim), kv[:, groups * maps * dim:].view(L, groups, vdim)
    first, scale = L - T, 2.0 * dim ** -0.5
    for i in (0, T // 2, T - 1):  # needles just outside and just inside of a query's window, and at the kept tokens' edge
        for place in (first + i - window, first + i - window + 1, keep - 1, keep):
            if 0 <= place <= first + i:
                for g in range(groups):
                    for m in range(maps):
                        k[place, g * maps + m] = 1.5 * q[i, g * (H // groups) + m]
    i, j = torch.arange(first, L)[:, None], torch.arange(L)[None, :]
    mask = (j <= i) & ((i - j < window) | (j < keep)) if window else j <= i
    qd, kd, vd = q.cpu().double(), k.cpu().double(), v.cpu().double()
    for out_dtype in (F32, BF16):
        out = torch.full((T, H * vdim), float("nan"), device=DEV, dtype=out_dtype)
        ops.window_attention(q, k, None, v, out, first_query=first, scale=scale, window=window, keep_first=keep, maps=maps)
        for h in range(H):
            g = h // (H // groups)
            s = (qd[:, h] @ kd[:, g * maps + h % maps].T * scale).masked_fill(~mask, -math.inf)
            near(out[:, h * vdim:(h + 1) * vdim], torch.softmax(s, -1) @ vd[:, g], 1e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,vdim,in_ld", [(1, 16, 16), (5, 40, 48), (3, 300, 304), (2, 7, 16)])
def test_map_difference(heads, vdim, in_ld, dtype):
    from tlaloc_b200 import ops

    rows, eps = 6, 1e-3
    w = {n: randn(16, seed=i, std=0.3).cpu().double() for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))}
    lam = math.exp(float((w["lq1"] * w["lk1"]).sum())) - math.exp(float((w["lq2"] * w["lk2"]).sum())) + 0.35
    a, gate = randn(rows, heads, 2, in_ld, seed=8), randn(rows, heads + 3, seed=9)
    out = torch.empty((rows, heads * vdim), device=DEV, dtype=dtype)
    want = oracle.difference(a.cpu().double()[..., :vdim], w.__getitem__, {"diff": 0.35}, eps)
    gated = (want * oracle.sigmoid(gate[:, 3:].cpu().double())[:, :, None]).reshape(rows, -1)
    kw = dict(rows=rows, heads=heads, vdim=vdim, in_ld=in_ld, lam=lam, keep=0.65, eps=eps)
    ops.map_difference(a, out, gate=gate[:, 3:], **kw)
    near(out, gated, 1e-5 if dtype == F32 else 8e-3)
    # as records of three slices, one of them empty for some rows
    rec = torch.zeros((3, rows, heads, 2, in_ld + 2), device=DEV)
    share = torch.rand((3, rows, heads, 2), generator=torch.Generator().manual_seed(1)).to(DEV) + 0.1
    share[1, ::2] = 0
    rec[..., 0] = randn(3, rows, heads, 2, seed=4, std=5.0)
    rec[..., 1] = share * torch.exp2(-rec[..., 0])
    rec[..., 2:] = a * rec[..., 1:2]
    rec[1, ::2, ..., 0], rec[1, ::2, ..., 2:] = -math.inf, float("nan")
    ops.map_difference(rec, out, slices=3, **kw)
    near(out, want.reshape(rows, -1), 2e-5 if dtype == F32 else 8e-3)


# ---------------------------------------------------------------------------------------------- retention

RETENTION = [(3, 20, 28, 12), (1, 4, 4, 2), (2, 64, 128, 64), (4, 128, 256, 128), (2, 16, 7, 0), (2, 256, 512, 256), (1, 300, 1000, 30)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,vdim,dims", RETENTION)
def test_retention_step(heads, dim, vdim, dims, dtype):
    """Three tokens of four sequences in slots of their own; the first starts from nothing, whatever its slot holds."""
    from tlaloc_b200 import ops
    from tlaloc_b200.rotary import Rotation, pair_tables

    T, eps, rot = 4, 1e-5, {"base": 300.0, "dims": dims}
    decay = [0.5 + 0.49 * (h + 1) / heads for h in range(heads)]
    cos, sin = (torch.from_numpy(t).to(DEV) for t in pair_tables(Rotation(dims, 300.0), 50))
    vp = -(-vdim // 4) * 4
    state = randn(7, heads, dim, vp, seed=1)
    state[3] = float("nan")
    slots, start = [3, 1, 6, 2], [0, 5, 17, 40]
    old = state.clone()
    x = randn(3, T, 2 * heads * (dim + vdim) + 4, seed=2)
    out = torch.empty((3, T, heads * vdim), device=DEV, dtype=dtype)
    for i in range(3):
        ops.retention_step(x[i, :, :2 * heads * (dim + vdim)], torch.tensor([p + i for p in start], dtype=torch.int32, device=DEV), cos, sin,
                           torch.tensor(decay, device=DEV), torch.tensor(slots, dtype=torch.int32, device=DEV), state, out[i], heads=heads, dim=dim, vdim=vdim,
                           rot_dims=dims, k_scale=dim ** -0.5, eps=eps)
    xd, hd, hv = x.cpu().double(), heads * dim, heads * vdim
    for t, (slot, p0) in enumerate(zip(slots, start)):
        rows = torch.zeros(p0 + 3, x.shape[2], dtype=torch.float64)
        rows[p0:] = xd[:, t]  # so that rotation counts from position 0
        turn = (lambda a: oracle.rotate_half(a, rot)) if dims else (lambda a: a)
        q = turn(rows[:, :hd].reshape(-1, heads, dim))[p0:]
        k = turn(rows[:, hd:2 * hd].reshape(-1, heads, dim))[p0:] * dim ** -0.5
        v, g = rows[p0:, 2 * hd:2 * hd + hv].reshape(-1, heads, vdim), rows[p0:, 2 * hd + hv:2 * (hd + hv)]
        o, s = oracle.recurrence(q, k, v, decay, None if p0 == 0 else old[slot, :, :, :vdim].cpu().double())
        near(out[:, t], oracle.rms(o, eps).reshape(3, -1) * oracle.silu(g), 1e-4 if dtype == F32 else 8e-3)
        near(state[slot, :, :, :vdim], s, 1e-5)
    for s in (0, 4, 5):
        assert torch.equal(state[s], old[s])


@pytest.mark.parametrize("heads,dim,vdim,dims,how,dtype", [(*r, how, dtype) for r in RETENTION for how, dtype in (("scan", F32), ("scan", BF16), ("chunks", BF16))
                                                           if how == "scan" or r[1] <= 256])
@pytest.mark.parametrize("tokens,fresh", [(2, True), (9, False), (130, True), (67, False), (64, False), (65, True), (700, False)])
def test_retention_over_a_portion(heads, dim, vdim, dims, tokens, fresh, how, dtype):
    from tlaloc_b200 import ops

    decay = [1 - 0.5 ** (3 + h) for h in range(heads)]
    vp, kd, vd = -(-vdim // 4) * 4, -(-dim // 16) * 16, -(-vdim // 16) * 16
    q, k, v = (torch.zeros((tokens, heads, n), device=DEV, dtype=dtype) for n in (kd, kd, vd))
    q[:, :, :dim], k[:, :, :dim], v[:, :, :vdim] = randn(tokens, heads, dim, seed=1), randn(tokens, heads, dim, seed=2, std=dim ** -0.5), randn(tokens, heads, vdim, seed=3)
    state = randn(4, heads, dim, vp, seed=4)
    if fresh:
        state[2] = float("nan")
    old = state.clone()
    o = torch.empty((tokens, heads, vdim), device=DEV)
    where = torch.full((tokens,), 2, dtype=torch.int32, device=DEV)
    positions = torch.arange(tokens, dtype=torch.int32, device=DEV) + (0 if fresh else 11)
    args = (q, k, v, positions, torch.tensor(decay, device=DEV), where, state, o)
    if how == "scan":
        ops.retention_scan(*args)
    else:
        scratch = torch.full((ops.retention_chunks_scratch_bytes(tokens, heads, dim, vdim) // 4,), float("nan"), device=DEV)
        ops.retention_chunks(*args, scratch)
    c = lambda t, n: t.cpu().double()[:, :, :n]
    want, s = oracle.recurrence(c(q, dim), c(k, dim), c(v, vdim), decay, None if fresh else old[2, :, :, :vdim].cpu().double())
    near(o, want, 5e-5)
    near(state[2, :, :, :vdim], s, 5e-5)
    assert torch.equal(state[[0, 1, 3]], old[[0, 1, 3]])
    gate, out = randn(tokens, heads * vdim + 4, seed=5), torch.empty((tokens, heads * vdim), device=DEV, dtype=dtype)
    ops.head_norm_gate(o, gate[:, 4:], out, 1e-5)
    near(out, oracle.rms(o.cpu().double(), 1e-5).reshape(tokens, -1) * oracle.silu(gate[:, 4:].cpu().double()), 2e-5 if dtype == F32 else 8e-3)
