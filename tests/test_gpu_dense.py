"""Dense matrices (KRONOS_CUDA_MATRIX_DENSE) through kronos_cuda_linear: the bf16 GEMV passes, the tensor-core GEMM and the
fp32 kernels against numpy, over sizes that are not multiples of any tile."""
import numpy as np
import pytest

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def ctx():
    import kronos_2t_b200 as k2
    c = k2.Context(0)
    yield c
    c.close()


def widen(b):
    return (b.astype(np.uint32) << 16).view(np.float32)


@pytest.mark.parametrize("rows,cols", [(8, 64), (100, 72), (640, 200), (1031, 1000), (384, 4096), (5000, 640)])
@pytest.mark.parametrize("n_tok", [1, 2, 3, 5, 8, 11, 16, 17, 33, 100, 300])
def test_bf16_products(ctx, rows, cols, n_tok):
    from kronos_2t_b200 import ffi
    rng = np.random.default_rng(rows * 7 + n_tok)
    w = ffi.bf16_bits(rng.standard_normal((rows, cols)).astype(np.float32))
    x = rng.standard_normal((n_tok, cols)).astype(np.float32)
    m = ctx.upload_dense(w, 16)
    got = ctx.linear(m, x)
    m.free()
    want = widen(ffi.bf16_bits(x)).astype(np.float64) @ widen(w).astype(np.float64).T
    err = np.abs(got - want).max() / np.sqrt(cols)
    assert err < 3e-5, (rows, cols, n_tok, err)


@pytest.mark.parametrize("rows,cols", [(5, 7), (100, 70), (641, 1000)])
@pytest.mark.parametrize("n_tok", [1, 3, 15, 16, 70])
def test_fp32_products(ctx, rows, cols, n_tok):
    rng = np.random.default_rng(rows + n_tok)
    w = rng.standard_normal((rows, cols)).astype(np.float32)
    x = rng.standard_normal((n_tok, cols)).astype(np.float32)
    m = ctx.upload_dense(w, 32)
    got = ctx.linear(m, x)
    m.free()
    err = np.abs(got - x.astype(np.float64) @ w.astype(np.float64).T).max() / np.sqrt(cols)
    assert err < 5e-6, err


def test_quantized_entry_points_refuse_dense_matrices(ctx):
    import kronos_2t_b200 as k2
    m = ctx.upload_dense(np.zeros((64, 64), np.uint16), 16)
    with pytest.raises(k2.KronosCudaError):
        ctx.gemv(m, np.zeros((1, 64), np.int8), np.ones((1, 1), np.float32), np.zeros((1, 1), np.int32))
    m.free()
