"""GPU tests of the single operations of the dense-weight decoders against plain PyTorch in float64."""
import math

import pytest
import torch

from tensorwarp_b200 import _dense

pytestmark = pytest.mark.gpu

DT = {torch.float32: _dense.TWM_DENSE_F32, torch.bfloat16: _dense.TWM_DENSE_BF16}


def gemm(a, w, epi, kernel, n, ldc=None):
    m, k = a.shape
    ldc = ldc or n
    out_dtype = torch.float32 if epi == _dense.EPI_STORE_F32 else a.dtype
    c = torch.full((m, ldc), 7.0, dtype=out_dtype, device="cuda")
    _dense.check(_dense.lib().twm_dense_gemm(DT[a.dtype], a.data_ptr(), a.stride(0), w.data_ptr(), w.stride(0), c.data_ptr(), ldc,
                                             m, n, k, epi, kernel, 0, torch.cuda.current_stream().cuda_stream), "gemm")
    torch.cuda.synchronize()
    assert _dense.device_error() == 0
    assert bool((c[:, n:] == 7.0).all()), "columns past N were written"
    return c[:, :n].double()


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


@pytest.mark.parametrize("m,n,k", [(1, 8, 16), (2, 48, 64), (5, 100, 80), (63, 130, 208), (128, 256, 512), (129, 257, 1040),
                                   (300, 1000, 336), (700, 2064, 128), (1024, 4096, 1024), (2100, 1530, 640)])
@pytest.mark.parametrize("epi", [_dense.EPI_STORE, _dense.EPI_STORE_F32, _dense.EPI_GELU_GLU])
@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2), (torch.bfloat16, 64),
                                          (torch.bfloat16, 128), (torch.bfloat16, 256), (torch.bfloat16, 512)])
def test_gemm(m, n, k, epi, dtype, kernel):
    gen = torch.Generator(device="cuda").manual_seed(m * 7 + n)
    a = torch.randn((m, k), generator=gen, device="cuda").to(dtype)
    w = (torch.randn((2 * n if epi == _dense.EPI_GELU_GLU else n, k), generator=gen, device="cuda") / math.sqrt(k)).to(dtype)
    got = gemm(a, w, epi, kernel, n, ldc=n + 3)
    ref = a.double() @ w.double().T
    if epi == _dense.EPI_GELU_GLU:
        ref = gelu_tanh(ref[:, :n]) * ref[:, n:]
    stored16 = dtype == torch.bfloat16 and epi != _dense.EPI_STORE_F32
    assert bool(((got - ref).abs() <= ref.abs() * (2 ** -8 if stored16 else 1e-5) + 3e-5).all())


def test_gemm_rows_with_longer_strides_and_no_bleed():
    """Operands inside wider buffers: what lies past K, past M and past N must not enter the result."""
    for dtype, kernel in ((torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2)):
        a = torch.full((200, 96), 1e30, device="cuda").to(dtype)
        w = torch.full((90, 112), 1e30, device="cuda").to(dtype)
        a[:70, :80] = torch.randn((70, 80), device="cuda").to(dtype)
        w[:66, :80] = torch.randn((66, 80), device="cuda").to(dtype)
        got = gemm(a[:70, :80], w[:66, :80], _dense.EPI_STORE_F32, kernel, 66)
        ref = a[:70, :80].double() @ w[:66, :80].double().T
        assert float((got - ref).abs().max()) < 1e-3
