"""Each kernel of the layered models against the plain restatement (lm_oracle.py), with inputs made so that a
key that is wrongly seen or missed, a lost sink or a wrong bias shows."""
import ctypes as C

import numpy as np
import pytest

import lm_oracle as lo

pytestmark = pytest.mark.gpu
RNG = lambda s: np.random.default_rng(s)


def up(a, dev):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a)).to(dev)


def sync():
    import torch
    torch.cuda.synchronize()


# ---- rows --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,dtype", [(64, "bf16"), (75, "bf16"), (1030, "f32")])
def test_embedding_with_position_vector(pkg, torch_dev, width, dtype):
    import torch
    table = torch.randn(50, width, device=torch_dev)
    table = table.bfloat16() if dtype == "bf16" else table
    tok, pos = np.array([3, 49, 0, 3, 7], np.int32), np.array([0, 1, 17, 5000, 70000], np.int32)
    freq = (10000.0 ** (-2.0 * np.arange(width // 2 + 1) / width)).astype(np.float32)
    d_tok, d_pos, d_freq = up(tok, torch_dev), up(pos, torch_dev), up(freq, torch_dev)
    for with_pos in (True, False):
        x = torch.full((5, width), 7.0, device=torch_dev)
        pkg.check(pkg.lib.cmlb200_embed_rows(table.data_ptr(), pkg.DT_BF16 if dtype == "bf16" else pkg.DT_F32, d_tok.data_ptr(), d_pos.data_ptr(),
                                             d_freq.data_ptr() if with_pos else None, 5, width, 50, x.data_ptr(), None))
        sync()
        want = table.float().cpu().numpy()[tok]
        if with_pos:
            want = want + lo.sinusoid(pos, width, np.float64)
        err = np.abs(x.cpu().numpy() - want).max(1)
        assert (err[:3] < 2e-6).all() and err[3] < 1e-3 and err[4] < 1e-2          # a 32-bit angle is good to p 2^-24


@pytest.mark.parametrize("dim,ldy,ldo", [(64, 64, 64), (75, 80, 128), (77, 77, 81), (5000, 5008, 5056)])
@pytest.mark.parametrize("out", ["bf16", "f32"])
def test_residual_norm_forms(pkg, torch_dev, dim, ldy, ldo, out):
    import torch
    rows, eps = 9, 1e-2
    g = torch.Generator(device=torch_dev).manual_seed(dim)
    x = torch.randn(rows, dim, device=torch_dev, generator=g) * 0.3
    y = torch.randn(rows, ldy, device=torch_dev, generator=g) * 0.1
    wp, wn = (1 + 0.5 * torch.randn(dim, device=torch_dev, generator=g) for _ in range(2))
    X, Y, P, N = (t.double().cpu().numpy() for t in (x, y[:, :dim], wp, wn))
    idx = up(np.array([8, 0, 3], np.int32), torch_dev)
    for case in ("post_next", "add_next", "post_only", "next_only", "gather"):
        xs = x.clone()
        o = torch.zeros(rows, ldo, device=torch_dev, dtype=torch.bfloat16 if out == "bf16" else torch.float32)
        has_y, n = case not in ("next_only", "gather"), 3 if case == "gather" else rows
        pkg.check(pkg.lib.cmlb200_residual_norm(xs.data_ptr(), y.data_ptr() if has_y else None, ldy, wp.data_ptr() if "post" in case else None,
                                                wn.data_ptr() if case != "post_only" else None, eps, n, dim, idx.data_ptr() if case == "gather" else None,
                                                o.data_ptr(), pkg.DT_BF16 if out == "bf16" else pkg.DT_F32, ldo, None))
        sync()
        want_x = X + (lo.rms_norm(Y, P, eps) if "post" in case else Y) if has_y else X
        assert np.abs(xs.cpu().numpy() - want_x).max() < 1e-5
        src = want_x[[8, 0, 3]] if case == "gather" else want_x
        got = o.float().cpu().numpy()
        want = lo.rms_norm(src, N, eps) if case != "post_only" else np.zeros((rows, dim))
        assert (np.abs(got[:n, :dim] - want) <= 2e-5 + (2.0 ** -8 * np.abs(want) if out == "bf16" else 0)).all()
        assert (got[:, dim:] == 0).all() and (got[n:] == 0).all()


@pytest.mark.parametrize("ff", [16, 33, 250])
@pytest.mark.parametrize("act", ["gelu", "silu"])
def test_glu_rows_f32(pkg, torch_dev, ff, act):
    import torch
    gu = torch.randn(3, 2 * ((ff + 15) // 16 * 16) + 8, device=torch_dev) * 2
    f = torch.zeros(3, ff + 3, device=torch_dev)
    pkg.check(pkg.lib.cmlb200_glu_rows_f32(gu.data_ptr(), gu.shape[1], 3, ff, pkg.ACT_GELU_TANH if act == "gelu" else pkg.ACT_SILU, f.data_ptr(), ff + 3, None))
    sync()
    a = gu.double().cpu().numpy()
    c = np.arange(ff) // 16 * 32 + np.arange(ff) % 16
    g, u = a[:, c], a[:, c + 16]
    want = (lo.gelu_tanh(g) if act == "gelu" else g / (1 + np.exp(-g))) * u
    assert np.abs(f.cpu().numpy()[:, :ff] - want).max() < 1e-5 and (f[:, ff:] == 0).all()


# ---- products ----------------------------------------------------------------------------------------------
def dense(pkg, torch_dev, w, dtype):
    """Padded device copy of a [rows, cols] fp32 array, and its descriptor."""
    import torch
    rows, cols = w.shape
    ld = (cols + 63) // 64 * 64
    full = np.zeros(((rows + 15) // 16 * 16, ld), np.float32)
    full[:rows, :cols] = w
    t = up(full, torch_dev)
    t = t.bfloat16() if dtype == pkg.DT_BF16 else t
    return t, pkg.Dense(dtype, rows, cols, ld, t.data_ptr())


def operand(torch_dev, x, dtype_bf16=True):
    import torch
    full = np.zeros((x.shape[0], (x.shape[1] + 63) // 64 * 64), np.float32)
    full[:, :x.shape[1]] = x
    t = up(full, torch_dev)
    return t.bfloat16() if dtype_bf16 else t


SHAPES = [(16, 64), (75, 75), (200, 144), (1000, 33), (130, 1111), (2064, 520)]


@pytest.mark.parametrize("N,K", SHAPES)
@pytest.mark.parametrize("M", [1, 2, 7, 8, 9, 16, 21, 32])
def test_decode_product(pkg, synth, torch_dev, N, K, M):
    import torch
    r = RNG(N + K + M)
    w, x = synth.bf16_round(r.standard_normal((N, K)))[1], synth.bf16_round(r.standard_normal((M, K)))[1]
    t, W = dense(pkg, torch_dev, w, pkg.DT_BF16)
    xd = operand(torch_dev, x)
    y = torch.full((M + 1, N + 5), 7.0, device=torch_dev)
    pkg.check(pkg.lib.cmlb200_gemv_dense(W, xd.data_ptr(), xd.shape[1], M, y.data_ptr(), N + 5, None))
    sync()
    got = y.cpu().numpy()
    assert np.abs(got[:M, :N] - x.astype(np.float64) @ w.T.astype(np.float64)).max() < 1e-5 * K ** 0.5 * 8
    assert (got[M] == 7).all() and (got[:, N:] == 7).all()


@pytest.mark.parametrize("N,K", SHAPES + [(512, 4096)])
@pytest.mark.parametrize("M", [1, 33, 128, 129, 300])
def test_prompt_product(pkg, synth, torch_dev, N, K, M):
    import torch
    r = RNG(N + K + M)
    w, x = synth.bf16_round(r.standard_normal((N, K)))[1], synth.bf16_round(r.standard_normal((M, K)))[1]
    t, W = dense(pkg, torch_dev, w, pkg.DT_BF16)
    xd = operand(torch_dev, x)
    y = torch.full((M + 1, N + 5), 7.0, device=torch_dev)
    pkg.check(pkg.lib.cmlb200_gemm_dense(W, xd.data_ptr(), xd.shape[1], M, y.data_ptr(), N + 5, None))
    sync()
    got = y.cpu().numpy()
    assert np.abs(got[:M, :N] - x.astype(np.float64) @ w.T.astype(np.float64)).max() < 1e-5 * K ** 0.5 * 8
    assert (got[M] == 7).all() and (got[:, N:] == 7).all()
    st = C.c_int(-1)
    pkg.check(pkg.lib.cmlb200_gemm_dense_status(C.byref(st), 1))
    assert st.value == 0


@pytest.mark.parametrize("M,N,K", [(2048, 4096, 4096), (4096, 2560, 1024), (700, 12288, 512)])
def test_prompt_product_many_tiles_per_cta(pkg, torch_dev, M, N, K):
    """More output tiles than SMs: the accumulators alternate and the operand ring runs on across tiles."""
    import torch
    x, w = (torch.randn(s, K, device=torch_dev).bfloat16() for s in (M, N))
    W = pkg.Dense(pkg.DT_BF16, N, K, K, w.data_ptr())
    y = torch.empty(M, N, device=torch_dev)
    for _ in range(5):
        y.zero_()
        pkg.check(pkg.lib.cmlb200_gemm_dense(W, x.data_ptr(), K, M, y.data_ptr(), N, torch.cuda.current_stream().cuda_stream))
        sync()
        want = x.float() @ w.float().T
        assert (y - want).abs().max().item() < 2e-3 * K ** 0.5


@pytest.mark.parametrize("ff,K", [(16, 64), (51, 75), (200, 144), (330, 700)])
@pytest.mark.parametrize("M", [1, 8, 13, 32, 33, 140])
@pytest.mark.parametrize("act", ["gelu", "silu"])
def test_gated_products(pkg, synth, torch_dev, ff, K, M, act):
    import torch
    r = RNG(ff + K + M)
    g, u = (synth.bf16_round(r.standard_normal((ff, K)) / K ** 0.5)[1] for _ in range(2))
    x = synth.bf16_round(r.standard_normal((M, K)))[1]
    rows = (ff + 15) // 16 * 32
    w = np.zeros((rows, K), np.float32)
    c = np.arange(ff) // 16 * 32 + np.arange(ff) % 16
    w[c], w[c + 16] = g, u
    t, W = dense(pkg, torch_dev, w, pkg.DT_BF16)
    xd = operand(torch_dev, x)
    code = pkg.ACT_GELU_TANH if act == "gelu" else pkg.ACT_SILU
    a, b = x.astype(np.float64) @ g.T, x.astype(np.float64) @ u.T
    want = (lo.gelu_tanh(a) if act == "gelu" else a / (1 + np.exp(-a))) * b
    for fn in ([pkg.lib.cmlb200_gemv_dense_glu] if M <= 32 else []) + [pkg.lib.cmlb200_gemm_dense_glu]:
        f = torch.zeros(M, ff + 6, device=torch_dev, dtype=torch.bfloat16)
        pkg.check(fn(W, xd.data_ptr(), xd.shape[1], M, ff, code, f.data_ptr(), ff + 6, None))
        sync()
        got = f.float().cpu().numpy()
        assert np.abs(got[:, :ff] - want).max() < 1e-2 * np.abs(want).max() and (got[:, ff:] == 0).all()


def test_product_f32_is_32_bit(pkg, torch_dev):
    import torch
    r = RNG(1)
    w, x = r.standard_normal((130, 777)).astype(np.float32), r.standard_normal((45, 777)).astype(np.float32)
    t, W = dense(pkg, torch_dev, w, pkg.DT_F32)
    xd = operand(torch_dev, x, False)
    y = torch.zeros(45, 131, device=torch_dev)
    pkg.check(pkg.lib.cmlb200_linear_dense_f32(W, xd.data_ptr(), xd.shape[1], 45, y.data_ptr(), 131, None))
    sync()
    assert np.abs(y.cpu().numpy()[:, :130] - x.astype(np.float64) @ w.T.astype(np.float64)).max() < 1e-4


def test_products_refuse_bad_arguments(pkg):
    fake, W = 0x10000, pkg.Dense(1, 64, 64, 64, 0x10000)
    lib = pkg.lib
    assert lib.cmlb200_gemv_dense(W, fake, 64, 33, fake, 64, None) == -1 and lib.cmlb200_gemv_dense(W, fake, 63, 1, fake, 64, None) == -1
    assert lib.cmlb200_gemv_dense(W, fake, 64, 1, fake, 63, None) == -1 and lib.cmlb200_gemm_dense(W, fake, 60, 40, fake, 64, None) == -1
    assert lib.cmlb200_gemm_dense_glu(W, fake, 64, 40, 33, 1, fake, 40, None) == -1
    assert lib.cmlb200_linear_dense_f32(W, fake, 64, 1, fake, 64, None) == -1
