"""Kernels of the hybrid families one at a time, against float64 statements of the same operator."""
import numpy as np
import pytest
import torch

from oracle import gutorax as G

pytestmark = pytest.mark.gpu

DTYPES = {"float32": (torch.float32, 2e-5), "bfloat16": (torch.bfloat16, 6e-3)}


def _rand(rng, *shape, scale=1.0, dtype=torch.bfloat16):
    """(device tensor, the float64 values it holds)"""
    t = torch.from_numpy((rng.standard_normal(shape) * scale).astype(np.float32)).to(dtype)
    return t.cuda(), t.double().numpy()


def _close(got, want, tol):
    got = got.double().cpu().numpy()
    assert np.isfinite(got).all()
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, err


def _dyt(rng, width):
    from cacheir_b200.hybrid_ops import DynamicTanh

    w, wn = _rand(rng, width, dtype=torch.float32)
    b, bn = _rand(rng, width, scale=0.2, dtype=torch.float32)
    return DynamicTanh(w, b, 0.6), lambda x: np.tanh(np.float64(np.float32(0.6)) * x) * wn + bn


@pytest.fixture(autouse=True)
def _status():
    yield
    from cacheir_b200 import hybrid_ops as H
    assert H.device_status() == 0


# ---- dense products ---------------------------------------------------------------------------------------------------
SHAPES = [(1, 8, 8), (3, 24, 40), (16, 136, 1024), (17, 256, 512), (33, 520, 2048), (64, 128, 4096), (65, 200, 72), (129, 640, 264),
          (300, 1000, 192), (520, 19072, 128)]


@pytest.mark.parametrize("t,n,k", SHAPES)
def test_dense_gemm_plain_float_and_activated(t, n, k):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(t + n + k)
    x, xn = _rand(rng, t, k)
    w, wn = _rand(rng, n, k, scale=k ** -0.5)
    want = xn @ wn.T
    f32 = torch.full((t, n), 9.0, device="cuda")
    H.dense_gemm(x, w, f32, epilogue=H.DENSE_F32)
    _close(f32, want, 1e-5)
    wide = torch.zeros((t, n + 8), device="cuda", dtype=torch.bfloat16)     # rows wider than the product stay untouched
    H.dense_gemm(x, w, wide)
    _close(wide[:, :n], want, 5e-3)
    assert float(wide[:, n:].abs().max()) == 0.0
    act = torch.empty((t, n), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, act, epilogue=H.DENSE_SILU, act_cols=n // 2 + 3)
    want_act = want.copy()
    want_act[:, :n // 2 + 3] = G.silu(want[:, :n // 2 + 3])
    _close(act, want_act, 5e-3)


@pytest.mark.parametrize("t,n,k", SHAPES)
def test_dense_gemm_geglu_and_gelu_embed(t, n, k):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(t * n)
    x, xn = _rand(rng, t, k)
    w, wn = _rand(rng, n, k, scale=1.5 * k ** -0.5)
    out = torch.empty((t, n // 2), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, out, epilogue=H.DENSE_GEGLU)
    y = xn @ wn.T
    _close(out, G.gelu_tanh(y[:, 0::2]) * y[:, 1::2], 6e-3)
    table, tn = _rand(rng, 11, n + 24)
    ids = torch.from_numpy(rng.integers(0, 11, t)).cuda()
    emb = torch.empty((t, n), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, emb, epilogue=H.DENSE_GELU_EMBED, ids=ids, table=table, table_col=16)
    _close(emb, G.gelu_tanh(y) * tn[ids.cpu().numpy(), 16:16 + n], 6e-3)


@pytest.mark.parametrize("nx", ["none", "copy", "dyt"])
@pytest.mark.parametrize("t,n,k", SHAPES)
def test_dense_gemm_finishes_a_sublayer(t, n, k, nx):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(n)
    x, xn = _rand(rng, t, k)
    w, wn = _rand(rng, n, k, scale=k ** -0.5)
    res, rn = _rand(rng, t, n, dtype=torch.float32)
    norm, f = _dyt(rng, n)
    norm2, f2 = _dyt(rng, n)
    out = torch.empty((t, n), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, epilogue=H.DENSE_RESIDUAL, residual=res, norm=norm,
                 nx={"none": None, "copy": H.Next(out), "dyt": H.Next(out, norm2)}[nx])
    want = rn + f(xn @ wn.T)
    _close(res, want, 1e-5)
    if nx != "none":
        _close(out, want if nx == "copy" else f2(want), 5e-3)


@pytest.mark.parametrize("t,batch,n,k,gap", [(1, 5, 40, 24, 16), (7, 3, 16, 48, 8), (40, 4, 136, 64, 0), (200, 2, 128, 512, 0)])
def test_dense_gemm_per_head_with_gate(t, batch, n, k, gap):
    from cacheir_b200 import hybrid_ops as H

    rng = np.random.default_rng(batch * n)
    x, xn = _rand(rng, t, batch * (k + gap))
    w, wn = _rand(rng, batch * n, k, scale=k ** -0.5)
    gate, gn = _rand(rng, t, batch * n + 8)
    heads = np.stack([xn[:, z * (k + gap):z * (k + gap) + k] @ wn[z * n:(z + 1) * n].T for z in range(batch)], axis=1)
    out = torch.empty((t, batch * n), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, out, epilogue=H.DENSE_GATED, batch=batch, x_batch_cols=k + gap, gate=gate)
    _close(out, heads.reshape(t, -1) * G.sigmoid(gn[:, :batch * n]), 6e-3)
    spaced = torch.zeros((t, batch * (n + 8)), device="cuda", dtype=torch.bfloat16)
    H.dense_gemm(x, w, spaced, batch=batch, x_batch_cols=k + gap, y_batch_cols=n + 8)
    _close(spaced.view(t, batch, n + 8)[:, :, :n], heads, 5e-3)
    assert float(spaced.view(t, batch, n + 8)[:, :, n:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("t,batch,n,k", [(1, 1, 1, 1), (5, 1, 77, 33), (130, 1, 65, 90), (9, 3, 7, 10)])
def test_dense_simple(t, batch, n, k, dtype):
    from cacheir_b200 import hybrid_ops as H

    td, tol = DTYPES[dtype]
    rng = np.random.default_rng(k)
    x, xn = _rand(rng, t, batch * k, dtype=td)
    w, wn = _rand(rng, batch * n, k, dtype=td)
    want = np.concatenate([xn[:, z * k:(z + 1) * k] @ wn[z * n:(z + 1) * n].T for z in range(batch)], axis=1)
    _close(H.dense_simple(x, w, torch.empty((t, batch * n), device="cuda", dtype=td), batch=batch, x_batch_cols=k), want, tol)
    _close(H.dense_simple(x, w, torch.empty((t, batch * n), device="cuda"), batch=batch, x_batch_cols=k), want, 2e-6)


def test_dense_gemm_refuses_what_it_cannot_take():
    from cacheir_b200 import hybrid_ops as H
    from cacheir_b200._lib import CacheIRB200Error

    x = torch.zeros((4, 20), device="cuda", dtype=torch.bfloat16)
    w = torch.zeros((8, 20), device="cuda", dtype=torch.bfloat16)
    out = torch.zeros((4, 8), device="cuda", dtype=torch.bfloat16)
    with pytest.raises(CacheIRB200Error):
        H.dense_gemm(x, w, out)
    with pytest.raises(ValueError):
        H.dense_gemm(x.float(), w, out)
    with pytest.raises(ValueError):
        H.dense_gemm(x, w, out.float())
    with pytest.raises(CacheIRB200Error):
        H.dense_gemm(x.cpu(), w, out)


# ---- row operators ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width", [(1, 1), (3, 90), (5, 128), (40, 2304)])
def test_row_operators(rows, width, dtype):
    from cacheir_b200 import hybrid_ops as H

    td, tol = DTYPES[dtype]
    rng = np.random.default_rng(width)
    norm, f = _dyt(rng, width)
    norm2, f2 = _dyt(rng, width)
    table, tn = _rand(rng, 13, width, dtype=td)
    ids = torch.from_numpy(rng.integers(0, 13, rows)).cuda()
    x = torch.empty((rows, width), device="cuda")
    out = torch.empty((rows, width), device="cuda", dtype=td)
    H.scaled_embedding(table, ids, x, 3.5, H.Next(out, norm))
    xn = tn[ids.cpu().numpy()] * 3.5
    _close(x, xn, 1e-6)
    _close(out, f(xn), tol)
    pick = torch.from_numpy(rng.integers(0, rows, rows + 2).astype(np.int32)).cuda()
    picked = torch.empty((rows + 2, width), device="cuda", dtype=td)
    _close(H.dyt_rows(x, norm2, picked, pick), f2(xn[pick.cpu().numpy()]), tol)
    y, yn = _rand(rng, rows, width, dtype=td)
    H.residual_dyt(x, y, norm, H.Next(out))
    xn = xn + f(yn)
    _close(x, xn, 2e-6)
    _close(out, xn, tol)
    w, wn = _rand(rng, width, dtype=torch.float32)
    H.residual_rms(x, y, w, 1e-3, H.Next(out, norm2))
    xn = xn + G.rms(yn, 1e-3) * wn
    _close(x, xn, 2e-6)
    _close(out, f2(xn), tol)
    H.residual_rms(x, y * 0, w, 1e-3)                      # a zero row stays finite through eps
    _close(x, xn, 2e-6)
    gate, gn = _rand(rng, rows, width + 4, dtype=td)
    got = H.gated_rms(y, gate[:, 3:3 + width], w, 1e-5, torch.empty_like(y))
    _close(got, G.rms(yn, 1e-5) * wn * G.sigmoid(gn[:, 3:3 + width]), tol)
    pair, pn = _rand(rng, rows, 2 * width, dtype=td)
    _close(H.glu_pairs(pair, torch.empty_like(y)), G.gelu_tanh(pn[:, 0::2]) * pn[:, 1::2], tol)
    side, sn = _rand(rng, 13, width + 7, dtype=td)
    _close(H.gelu_embed(y, ids, side, 5, torch.empty_like(y)), G.gelu_tanh(yn) * sn[ids.cpu().numpy(), 5:5 + width], tol)
    z = y.clone()
    H.silu_cols(z, width - width // 3)
    want = yn.copy()
    want[:, :width - width // 3] = G.silu(yn[:, :width - width // 3])
    _close(z, want, tol)
