"""Unquantized projections through the C ABI against a plain f64 product: the f32 and bf16 paths, the tensor-core kernel's row
classes and K slices, edges of every tile, strided and batched operands, bias, squared ReLU, residual in place (needs a B200)."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


@pytest.fixture(autouse=True)
def no_wait_runs_out():
    """Every device-side wait is bounded; one that runs out leaves a status word (and a wrong result)."""
    yield
    from tlaloc_b200 import _native

    torch.cuda.synchronize()
    assert _native.lib().tlaloc_b200_device_status() == 0


def reference(x, w, bias=None, residual=None, relu2=False):
    y = x.double() @ w.double().transpose(-1, -2)
    if bias is not None:
        y = y + bias.double()
    if relu2:
        y = y.clamp_min(0) ** 2
    return y if residual is None else y + residual.double()


def rand(*shape, dtype=torch.bfloat16, seed=0):
    g = torch.Generator(device=DEV)
    g.manual_seed(seed + sum(shape))
    return torch.randn(shape, device=DEV, generator=g).to(dtype)


def close(got, want, k, f32_out=True):
    scale = float(want.abs().max())
    tol = (2e-6 * np.sqrt(k) if f32_out else 8e-3) * max(scale, 1.0)
    err = float((got.double() - want).abs().max())
    assert err <= tol, (err, tol)


@pytest.mark.parametrize("m", [1, 3, 31, 32, 33, 64, 100, 128, 129, 256, 300, 1000])
@pytest.mark.parametrize("n,k", [(128, 64), (200, 136), (96, 24), (1030, 520)])
def test_bf16_row_classes_and_edges(m, n, k):
    from tlaloc_b200 import ops

    x, w, b, r = rand(m, k), rand(n, k, seed=1), rand(n, dtype=torch.float32, seed=2), rand(m, n, dtype=torch.float32, seed=3)
    y = torch.empty((m, n), device=DEV)
    ops.dense_gemm(ops.dense(x, w, y))
    close(y, reference(x, w), k)
    y16 = torch.empty((m, n), device=DEV, dtype=torch.bfloat16)
    ops.dense_gemm(ops.dense(x, w, y16, bias=b, act=1), weights_const=True)
    close(y16, reference(x, w, b, relu2=True), k, False)
    want = reference(x, w, b, r)
    ops.dense_gemm(ops.dense(x, w, r, bias=b, residual=r))  # the residual stream in place
    close(r, want, k)


@pytest.mark.parametrize("m", [1, 20, 60, 120])
def test_long_k_runs_in_slices(m):
    from tlaloc_b200 import ops

    x, w = rand(m, 18432), rand(512, 18432, seed=1)
    y = torch.empty((m, 512), device=DEV)
    ops.dense_gemm(ops.dense(x, w, y), weights_const=True)
    close(y, reference(x, w), 18432)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [1, 37, 130, 600])
def test_two_problems_strided_outputs(dtype, m):
    """Two inputs, two weights, one launch; the second result lands in columns of a wider matrix and nowhere else."""
    from tlaloc_b200 import ops

    x1, x2, w1, w2 = rand(m, 320, dtype=dtype), rand(m, 320, dtype=dtype, seed=1), rand(232, 320, dtype=dtype, seed=2), rand(704, 320, dtype=dtype, seed=3)
    y1, wide = torch.empty((m, 232), device=DEV), torch.full((m, 1000), 7.0, device=DEV, dtype=dtype)
    ops.dense_gemm(ops.dense(x1, w1, y1), ops.dense(x2, w2, wide[:, 96:800], act=1))
    close(y1, reference(x1, w1), 320)
    close(wide[:, 96:800], reference(x2, w2, relu2=True), 320, dtype == torch.float32)
    assert bool((wide[:, :96] == 7).all()) and bool((wide[:, 800:] == 7).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m,heads,k,n", [(1, 5, 40, 72), (9, 3, 32, 128), (70, 4, 64, 48), (300, 3, 24, 136), (64, 16, 512, 128)])
def test_a_batch_of_heads_in_interleaved_rows(dtype, m, heads, k, n):
    """x and y hold a row's heads side by side: [rows, heads, ...] seen as one problem per head."""
    from tlaloc_b200 import ops

    x, w = rand(m, heads, k + 8, dtype=dtype), rand(heads, n, k, dtype=dtype, seed=1)
    y = torch.full((m, heads, n + 16), 3.0, device=DEV, dtype=dtype)
    ops.dense_gemm(ops.dense(x[:, :, :k].transpose(0, 1), w, y[:, :, :n].transpose(0, 1)))
    want = torch.einsum("mhk,hnk->mhn", x[:, :, :k].double(), w.double())
    close(y[:, :, :n], want, k, dtype == torch.float32)
    assert bool((y[:, :, n:] == 3).all())


def test_unaligned_operands_take_the_plain_kernel():
    from tlaloc_b200 import ops

    wide, w = rand(33, 131), rand(50, 77, seed=1)
    y = torch.empty((33, 50), device=DEV)
    ops.dense_gemm(ops.dense(wide[:, 3:80], w, y))
    close(y, reference(wide[:, 3:80], w), 77)


def test_f32_is_true_f32():
    """Values that bf16 or a 10-bit mantissa would round away survive."""
    from tlaloc_b200 import ops

    x = torch.full((4, 64), 1.0 + 2.0 ** -20, device=DEV)
    w = torch.zeros((8, 64), device=DEV)
    w[:, 0], w[:, 1] = 1.0, -1.0
    x[:, 1] = 1.0
    y = torch.empty((4, 8), device=DEV)
    ops.dense_gemm(ops.dense(x, w, y))
    assert bool((y == 2.0 ** -20).all())


def test_bad_arguments_are_refused():
    from tlaloc_b200 import ops

    x, w, y = rand(4, 64), rand(8, 64), torch.empty((4, 8), device=DEV)
    for bad in (lambda: ops.dense(x.cpu(), w, y), lambda: ops.dense(x[:, :32], w, y), lambda: ops.dense(x, w, y.t()),
                lambda: ops.dense(x.float(), w, y), lambda: ops.dense(x, w, y, bias=torch.zeros(7, device=DEV)),
                lambda: ops.dense(x, w, y, residual=torch.zeros((4, 8), device=DEV, dtype=torch.bfloat16))):
        with pytest.raises(ValueError):
            bad()
