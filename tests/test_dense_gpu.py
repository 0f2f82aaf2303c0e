"""fb_dense - activations by bf16 weights whose output columns each lie together - with each of its epilogues, against the
same arithmetic in fp32 torch on the CPU, and the planner's choice of it: the expressions a model writes, fused, agree with
the same expressions computed op by op."""
import numpy as np
import pytest
import torch

from ferrite_b200 import _lib, ops

pytestmark = pytest.mark.gpu

# tokens x K x N: one tile and many, K within a step, K split over a cluster, tokens past a tile, ragged edges everywhere
SHAPES = [(1, 64, 128), (3, 40, 72), (16, 512, 96), (17, 264, 200), (33, 1536, 384), (128, 96, 1000), (200, 576, 130), (300, 2048, 256), (513, 320, 4608), (5, 4096, 512)]


def rand(*shape, seed=0, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16()


def close(got, want, rel):
    err = (got.float().cpu() - want).abs().max() / want.abs().max()
    assert err <= rel, float(err)


@pytest.mark.parametrize("M,K,N", SHAPES)
@pytest.mark.parametrize("settled", [False, True])
def test_plain(cuda, M, K, N, settled):
    x, w = rand(M, K, seed=1), rand(N, K, seed=2, scale=K ** -0.5)
    want = x.float() @ w.float().T
    xd, wd = x.to(cuda)[None], w.to(cuda)[None]
    torch.cuda.synchronize()
    for dtype, rel in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        out = torch.full((1, M, N + 8), 7.0, dtype=dtype, device=cuda)
        ops.dense(xd, wd.transpose(1, 2), out[:, :, :N], settled)
        close(out[0, :, :N], want, rel)
        assert (out[0, :, N:] == 7).all(), "nothing written beside the result"
        again = torch.empty_like(out)[:, :, :N]
        ops.dense(xd, wd.transpose(1, 2), again, settled)
        assert torch.equal(again, out[:, :, :N]), "the same bits every run"


@pytest.mark.parametrize("M", [1, 30, 270])
@pytest.mark.parametrize("B,K,N", [(3, 48, 80), (40, 128, 512), (7, 512, 56)])
def test_batch_and_gate(cuda, M, B, K, N):
    # entries interleaved in the rows, as heads are: x [M, B (K + 8)], out [M, B N]
    x, w, g = rand(M, B, K + 8, seed=3).to(cuda), rand(B, N, K, seed=4, scale=K ** -0.5).to(cuda), torch.randn(M, B + 5, generator=torch.Generator().manual_seed(5)).to(cuda)
    out = torch.empty(M, B, N, dtype=torch.bfloat16, device=cuda)
    xs = x[:, :, :K].permute(1, 0, 2)
    want = torch.einsum("mbk,bnk->mbn", x[:, :, :K].float().cpu(), w.float().cpu())
    ops.dense(xs, w.transpose(1, 2), out.permute(1, 0, 2))
    close(out, want, 5e-3)
    ops.dense(xs, w.transpose(1, 2), out.permute(1, 0, 2), kind=_lib.DENSE_GATE, gate=g.data_ptr(), ld_gate=g.stride(0))
    close(out, want * torch.sigmoid(g.cpu()[:, :B, None]), 5e-3)


@pytest.mark.parametrize("M,K,N", [(1, 256, 64), (20, 96, 416), (130, 1024, 1056), (300, 264, 160)])
def test_silu_and_gated_unit(cuda, M, K, N):
    x, w = rand(M, K, seed=6), rand(N, K, seed=7, scale=3 * K ** -0.5)
    acc = x.float() @ w.float().T
    xd, wt = x.to(cuda)[None], w.to(cuda)[None].transpose(1, 2)
    for n in (0, N // 3, N):
        out = torch.empty(1, M, N, dtype=torch.bfloat16, device=cuda)
        ops.dense(xd, wt, out, kind=_lib.DENSE_SILU, act_cols=n)
        want = acc.clone()
        want[:, :n] = torch.nn.functional.silu(want[:, :n])
        close(out[0], want, 5e-3)
    limit, slope = 1.5, 1.3
    out = torch.empty(1, M, N // 2, dtype=torch.bfloat16, device=cuda)
    ops.dense(xd, wt, out, kind=_lib.DENSE_GLU, limit=limit, slope=slope)
    g, u = acc[:, :N // 2].clamp(max=limit), acc[:, N // 2:].clamp(-limit, limit)
    close(out[0], g * torch.sigmoid(slope * g) * (u + 1), 5e-3)


@pytest.mark.parametrize("M,K,N", [(1, 256, 192), (9, 1024, 200), (64, 4096, 256), (300, 96, 136)])
def test_dynamic_tanh_and_add(cuda, M, K, N):
    x, w = rand(M, K, seed=8), rand(N, K, seed=9, scale=K ** -0.5)
    gen = torch.Generator().manual_seed(10)
    v = lambda: torch.randn(N, generator=gen)
    res, w1, b1, w2, b2, a1, a2 = torch.randn(M, N, generator=gen), v(), v(), v(), v(), torch.tensor([0.7]), torch.tensor([0.4])
    want = res + torch.tanh(0.7 * (x.float() @ w.float().T)) * w1 + b1
    d = [t.to(cuda) for t in (res, w1, b1, w2, b2, a1, a2)]
    for hand in (False, True):
        out, h = torch.empty(1, M, N, device=cuda), torch.empty(M, N, dtype=torch.bfloat16, device=cuda)
        extra = dict(h_out=h.data_ptr(), ld_h=N, alpha2=d[6].data_ptr(), w2=d[3].data_ptr(), b2=d[4].data_ptr()) if hand else {}
        ops.dense(x.to(cuda)[None], w.to(cuda)[None].transpose(1, 2), out, kind=_lib.DENSE_DYT_ADD, residual=d[0].data_ptr(), ld_residual=N, alpha=d[5].data_ptr(),
                  w=d[1].data_ptr(), b=d[2].data_ptr(), **extra)
        close(out[0], want, 2e-5)
        if hand:
            close(h, torch.tanh(0.4 * want) * w2 + b2, 5e-3)


def test_the_planner_fuses_what_a_layer_writes(cuda):
    from ferrite_b200 import mixers, tensor
    from ferrite_b200.tensor import Runtime, Tensor
    rt = Runtime(0)
    M, D, F = 37, 192, 96
    rng = np.random.default_rng(11)
    turned = lambda n, k: Tensor.of(rt, rng.normal(0, k ** -0.5, (n, k))).T
    vec = lambda n=D, at=0.0: Tensor.of(rt, at + rng.normal(0, 0.3, (1, n)), "fp32")
    p = {"gate_up": turned(2 * F, D), "down": turned(D, F)} | {n + s: vec(1, 0.6) if s == ".alpha" else vec() for n in ("n1", "n2", "n3") for s in ("", ".b", ".alpha")}
    x0 = rng.normal(0, 1, (M, D)).astype(np.float32)

    def run():
        x = Tensor.of(rt, x0, "fp32")
        h = mixers.dyt(x, p, "n1").cast("bf16")
        x = x + mixers.dyt(mixers.clamped_mlp(h, p, "", 1.2, 1.7), p, "n2")
        h = mixers.dyt(x, p, "n3").cast("bf16").realize()
        return x.realize().numpy()[0], h.numpy()[0]
    before = rt.launches
    fused = run()
    names = [n for n, _ in rt.profile(before)]
    assert "dense glu" in names and "dense dyt add" in names and sum(n == "elementwise" for n in names) == 1, names
    supports, ops.dense_supports = ops.dense_supports, lambda *a: False
    try:
        plain = run()
    finally:
        ops.dense_supports = supports
    for f, g in zip(fused, plain):
        assert np.abs(f - g).max() < 0.02 * np.abs(g).max()
