"""bf16 products (gptb200_linear_bf16) against fp32 products of the same bf16 values: every output form on every kernel."""
import ctypes

import pytest
import torch

pytestmark = pytest.mark.gpu

# rows x columns x k: single rows, the weight-streaming kernel's limits, one-CTA tiles, split k, CTA pairs (whole tiles and cut ranges)
SHAPES = [(1, 64, 64), (1, 768, 3072), (1, 2048, 4104), (1, 4160, 1032), (3, 320, 72), (8, 1088, 4096), (9, 64, 8), (17, 192, 200), (100, 576, 1032), (129, 64, 64), (300, 1536, 768), (1000, 320, 512), (2048, 2048, 1024),
          (2500, 2944, 2048), (257, 4096, 4096)]


def gelu(z):
    return torch.nn.functional.gelu(z, approximate="tanh")


@pytest.fixture(scope="module")
def backend():
    import gpt_b200
    from gpt_b200 import decoder
    be = gpt_b200.Backend(0, torch.cuda.current_stream().cuda_stream)
    decoder.load_library()
    yield be
    be.close()


def run(be, kind, out, x, w, n, tail=None, tail_col=1 << 30, factor=None, rows=None):
    from gpt_b200 import decoder
    p = lambda t: ctypes.c_void_p(t.data_ptr()) if t is not None else None
    rc = decoder.load_library().gptb200_linear_bf16(be.handle, kind, p(out), out.stride(0), p(x), x.stride(0), p(w), x.shape[0], n, w.shape[1], p(tail), tail_col,
                                                    tail.stride(0) if tail is not None else 0, p(factor), p(rows), factor.stride(0) if factor is not None else 0)
    assert rc == 0, be.lib.gptb200_last_error(be.handle)
    be.synchronize()


def close(got, want, tol):
    assert torch.isfinite(got).all()
    assert (got.float() - want).abs().max() <= tol * want.abs().max()


@pytest.mark.parametrize("m,n,k", SHAPES)
def test_forms(backend, m, n, k):
    torch.manual_seed(m * 7 + n + k)
    big = torch.randn(m, k + 24, device="cuda").bfloat16()
    x = big[:, 8:8 + k]                                     # a slice of wider rows
    w = (torch.randn(n, k, device="cuda") / k ** 0.5).bfloat16()
    ref = x.float().double() @ w.double().T
    ref = ref.float()
    guard = lambda rows, cols, dt: torch.full((rows + 1, cols), 77.0, device="cuda", dtype=dt)
    out = guard(m, n, torch.float32)
    run(backend, 0, out, x, w, n)
    close(out[:m], ref, 1e-5)
    assert (out[m] == 77).all()
    wide = guard(m, n + 16, torch.float32)                  # row pitch larger than the columns
    run(backend, 0, wide, x, w, n)
    close(wide[:m, :n], ref, 1e-5)
    assert (wide[:, n:] == 77).all() and (wide[m] == 77).all()
    out = guard(m, n + 8, torch.bfloat16)
    run(backend, 1, out, x, w, n)
    close(out[:m, :n], ref, 5e-3)
    assert (out[:, n:] == 77).all() and (out[m] == 77).all()
    cut = n // 2 // 32 * 32
    out, tail = guard(m, cut + 8, torch.bfloat16), guard(m, n - cut + 3, torch.float32)
    run(backend, 1, out, x, w, n, tail=tail, tail_col=cut)
    close(out[:m, :cut], ref[:, :cut], 5e-3)
    close(tail[:m, :n - cut], ref[:, cut:], 1e-5)
    assert (out[:, cut:] == 77).all() and (out[m] == 77).all() and (tail[:, n - cut:] == 77).all() and (tail[m] == 77).all()
    g = ref.view(m, n // 64, 2, 32)
    out = guard(m, n // 2 + 8, torch.bfloat16)
    run(backend, 2, out, x, w, n)
    close(out[:m, :n // 2], (gelu(g[:, :, 0]) * g[:, :, 1]).reshape(m, n // 2), 5e-3)
    assert (out[:, n // 2:] == 77).all() and (out[m] == 77).all()
    out = guard(m, n // 2 + 8, torch.bfloat16)
    run(backend, 4, out, x, w, n)
    close(out[:m, :n // 2], (torch.nn.functional.silu(g[:, :, 0]) * g[:, :, 1]).reshape(m, n // 2), 5e-3)
    assert (out[:, n // 2:] == 77).all() and (out[m] == 77).all()
    factor = torch.randn(13, n + 8, device="cuda").bfloat16()
    rows = torch.randint(0, 13, (m,), device="cuda", dtype=torch.int32)
    out = guard(m, n + 8, torch.bfloat16)
    run(backend, 3, out, x, w, n, factor=factor, rows=rows)
    close(out[:m, :n], gelu(ref) * factor[rows.long(), :n].float(), 5e-3)
    assert (out[:, n:] == 77).all() and (out[m] == 77).all()


@pytest.mark.parametrize("option,value", [("pair", 1), ("pair", -1), ("stream_k", 1), ("tile_n", 256), ("tile_n", 128), ("max_splits", 4), ("gemv_rows", 0)])
def test_forced_kernels(backend, option, value):
    torch.manual_seed(3)
    backend.set_option(option, value)
    try:
        for m, n, k in ((5, 384, 640), (513, 896, 768), (640, 640, 2048)):
            x, w = torch.randn(m, k, device="cuda").bfloat16(), (torch.randn(n, k, device="cuda") / k ** 0.5).bfloat16()
            ref = (x.double() @ w.double().T).float()
            out = torch.empty(m, n, device="cuda")
            run(backend, 0, out, x, w, n)
            close(out, ref, 1e-5)
            g = ref.view(m, n // 64, 2, 32)
            half = torch.empty(m, n // 2, device="cuda", dtype=torch.bfloat16)
            run(backend, 2, half, x, w, n)
            close(half, (gelu(g[:, :, 0]) * g[:, :, 1]).reshape(m, n // 2), 5e-3)
    finally:
        backend.set_option(option, 8 if option == "gemv_rows" else 0)


def test_wrong_sizes_are_refused(backend):
    from gpt_b200 import decoder
    lib = decoder.load_library()
    t = torch.zeros(64, 64, device="cuda", dtype=torch.bfloat16)
    p = ctypes.c_void_p(t.data_ptr())
    args = lambda kind, n, k, pitch: (backend.handle, kind, p, 64, p, pitch, p, 4, n, k, None, 1 << 30, 0, None, None, 0)
    assert lib.gptb200_linear_bf16(*args(0, 64, 60, 64)) == 1       # k not a multiple of 8
    assert lib.gptb200_linear_bf16(*args(0, 64, 64, 60)) == 1       # pitch
    assert lib.gptb200_linear_bf16(*args(2, 96, 64, 64)) == 1       # gated columns
    assert lib.gptb200_linear_bf16(*args(4, 96, 64, 64)) == 1
    assert lib.gptb200_linear_bf16(*args(3, 64, 64, 64)) == 1       # no factor
    assert lib.gptb200_linear_bf16(*args(7, 64, 64, 64)) == 1       # kind
