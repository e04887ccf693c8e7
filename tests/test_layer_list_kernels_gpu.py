"""Kernels of the layer-list architectures through the C ABI, each against a plain fp32 / fp64 computation."""

import ctypes as C

import numpy as np
import pytest
import torch

import fegenex_oracle as fo
from q38_testlib import pkg

pytestmark = pytest.mark.gpu


def up(x, to):
    return (x + to - 1) // to * to


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to("cuda", dtype)


def bf16(a):
    return torch.as_tensor(np.asarray(a)).to(torch.bfloat16).to(torch.float64).numpy()


class DenseWeight:
    """W [n][k] and bias on the device in the padded layout the kernels take."""

    def __init__(self, w, bias=None):
        n, k = w.shape
        self.ld = up(k, 64)
        self.w = torch.zeros((up(n, 16), self.ld), dtype=torch.bfloat16, device="cuda")
        self.w[:n, :k] = dev(w, torch.bfloat16)
        self.b = None
        if bias is not None:
            self.b = torch.zeros(up(n, 16), dtype=torch.float32, device="cuda")
            self.b[:n] = dev(bias)
        self.desc = pkg.DenseWeight(pkg.ptr(self.w), pkg.ptr(self.b), n, k, self.ld)


def run_gemm(x, w, kind, out_cols, act, config=-1, ldo=None):
    m, k = x.shape
    tdt = torch.bfloat16 if act == pkg.ACT_BF16 else torch.float32
    ldx, ldo = up(k, 64), ldo or out_cols
    xd = torch.zeros((m, ldx), dtype=tdt, device="cuda")
    xd[:, :k] = dev(x, tdt)
    out = torch.full((m, ldo), 7.0, dtype=torch.float32 if kind == pkg.DENSE_STORE_F32 else tdt, device="cuda")
    ep = pkg.DenseEpilogue(kind, pkg.ptr(out), ldo)
    pkg.check(pkg.kernels().q38_dense_gemm(pkg.ptr(xd), ldx, act, m, C.byref(w.desc), C.byref(ep), None, None, config))
    torch.cuda.synchronize()
    assert pkg.kernels().q38_device_error(1) == 0
    return out.double().cpu().numpy()


@pytest.mark.parametrize("n,k", [(384, 256), (200, 72), (96, 1000), (1042, 520), (16, 8)])
@pytest.mark.parametrize("m", [1, 5, 16, 17, 40, 130, 300])
def test_dense_gemm_every_kernel(n, k, m):
    rng = np.random.default_rng(n + k + m)
    x, wt, b = bf16(rng.standard_normal((m, k))), bf16(rng.standard_normal((n, k)) / np.sqrt(k)), rng.standard_normal(n)
    w = DenseWeight(wt, b)
    want = x @ wt.T + b.astype(np.float32)
    names = [pkg.kernels().q38_dense_gemm_config_name(i).decode() for i in range(pkg.kernels().q38_dense_gemm_num_configs())]
    for i, name in [(-1, "auto")] + list(enumerate(names)):
        if "cluster" in name and (k + 63) // 64 < int(name[-1]):
            continue
        got = run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i, ldo=n + 3)
        assert np.all(got[:, n:] == 7.0)
        assert np.abs(got[:, :n] - want).max() < 2e-4, name
        got = run_gemm(x, w, pkg.DENSE_STORE, n, pkg.ACT_BF16, i, ldo=n + 6)
        assert np.all(got[:, n:] == 7.0)
        assert np.all(np.abs(got[:, :n] - want) < 2e-4 + np.abs(want) / 256), name
        again = run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i)
        assert np.array_equal(again, run_gemm(x, w, pkg.DENSE_STORE_F32, n, pkg.ACT_BF16, i)), name
        for kind, act in ((pkg.DENSE_GLU_GELU, fo.gelu_tanh), (pkg.DENSE_GLU_SILU, fo.silu)):
            got = run_gemm(x, w, kind, n // 2, pkg.ACT_BF16, i)
            product = act(want[:, 0::2]) * want[:, 1::2]
            assert np.all(np.abs(got - product) < 1e-3 + np.abs(product) / 256), name
    x32 = rng.standard_normal((m, k))
    got = run_gemm(x32, w, pkg.DENSE_STORE, n, pkg.ACT_F32)
    assert np.abs(got - (x32.astype(np.float32).astype(np.float64) @ wt.T + b)).max() < 1e-5
