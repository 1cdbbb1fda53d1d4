"""The product of few rows whose clusters share K, against a float64 product."""
import pytest
import torch

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _rel(a, b):
    return float((a.double().cpu() - b).norm() / (b.norm() + 1e-30))


@pytest.mark.parametrize("M", [1, 2, 15, 16, 17, 40, 64, 65, 128])
@pytest.mark.parametrize("N,K", [(128, 512), (3072, 2048), (2048, 5632), (100, 72), (1000, 136), (37, 4096), (8192, 64), (16, 8), (11264, 256)])
def test_few_rows_of_every_size(M, N, K):
    from rumus_b200.ops import native
    torch.manual_seed(M + N)
    a, w = torch.randn(M, K + 8).to(BF)[:, :K], torch.randn(N, K).to(BF)
    want = a.double() @ w.double().T
    ag, wg = torch.empty(M, K + 8, dtype=BF, device="cuda")[:, :K].copy_(a), w.cuda()
    out = torch.full((M, N + 5), 7.0, dtype=F32, device="cuda")
    native.gemm(ag, wg.t(), out=out[:, :N], out_dtype=F32, path=4)
    assert native.gemm.last_path == 4
    assert _rel(out[:, :N], want) < 1e-5 and bool((out[:, N:] == 7).all())
    assert _rel(native.gemm(ag, wg.t(), path=4), want) < 3e-3
    assert native.read_status() == 0


@pytest.mark.parametrize("act,fn", [(None, lambda v: v), ("relu", torch.relu), ("relu2", lambda v: torch.relu(v) ** 2),
                                    ("silu", torch.nn.functional.silu), ("gelu", lambda v: torch.nn.functional.gelu(v, approximate="tanh"))])
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("M,N,K", [(3, 1024, 1024), (50, 300, 2048)])
def test_epilogue_terms(act, fn, f32, M, N, K):
    from rumus_b200.ops import native
    torch.manual_seed(N)
    a, w, bias = torch.randn(M, K).to(BF), (torch.randn(N, K) * K ** -0.5).to(BF), torch.randn(N).to(BF)
    res = torch.randn(M, N).to(F32 if f32 else BF)
    got = native.gemm(a.cuda(), w.cuda().t(), bias=bias.cuda(), act=act, residual=res.cuda(), alpha=0.7, out_dtype=F32 if f32 else BF)
    assert native.gemm.last_path == 4
    want = fn(0.7 * (a.double() @ w.double().T) + bias.double()) + res.double()
    assert _rel(got, want) < (2e-6 if f32 else 3e-3)


def test_sums_do_not_depend_on_the_other_rows():
    """A row's numbers are the same bits alone and among others of the same tile size."""
    from rumus_b200.ops import native
    torch.manual_seed(0)
    a, w = torch.randn(16, 2048).to(BF).cuda(), torch.randn(2048, 2048).to(BF).cuda()
    whole = native.gemm(a, w.t(), out_dtype=F32)
    for i in (0, 7, 15):
        assert torch.equal(native.gemm(a[i:i + 1], w.t(), out_dtype=F32)[0], whole[i])
