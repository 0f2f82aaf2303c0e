"""The kernels of attention over cached latents and of linear attention with decay, one by one, through the C ABI, against
float64 numpy (oracle/binutar.py's functions where they fit): bf16 sizes the tensor-core kernels take, and fp32 and odd
sizes, which run elsewhere."""
import numpy as np
import pytest
import torch

from ferrite_b200 import ops
from oracle import binutar as oracle

pytestmark = pytest.mark.gpu
f64 = np.float64


def draw(rng, *shape, dtype=torch.bfloat16, scale=1.0):
    return torch.from_numpy((rng.normal(0, 1, shape) * scale).astype(np.float32)).to(dtype)


def attend(q, cache, rank, first, last, scale, sink):
    """q [T, H, W] over cache rows first[t] .. first[t] + last[t]."""
    out = np.zeros((*q.shape[:2], rank))
    for t in range(q.shape[0]):
        k = cache[first[t]:first[t] + last[t] + 1]
        s = np.einsum("hw,kw->hk", q[t], k) * scale
        m = s.max(1, keepdims=True) if sink is None else np.maximum(s.max(1), sink)[:, None]
        e = np.exp(s - m)
        total = e.sum(1) + (0 if sink is None else np.exp(sink - m[:, 0]))
        out[t] = e @ k[:, :rank] / total[:, None]
    return out


# heads, latent, turned part: one row tile and several, a latent of one 64-column piece up to the widest, pieces cut short
SIZES = [(12, 128, 48), (3, 64, 16), (20, 96, 24), (16, 512, 64), (40, 256, 32), (80, 192, 8), (64, 512, 64), (1, 40, 8), (5, 33, 7), (4, 600, 40)]


@pytest.mark.parametrize("H,rank,rot", SIZES)
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_decode_over_sequences_of_unequal_length(cuda, H, rank, rot, dtype):
    rng = np.random.default_rng(1)
    T, part, W = 5, 704, rank + rot
    cache = draw(rng, T * part, W, dtype=dtype)
    base = np.array([3, 0, 2, 4, 1], np.int32) * part
    last = np.array([0, 63, 64, 700, 317], np.int32)
    q = draw(rng, T, H * W, dtype=dtype)
    qv, cv = q.float().numpy().astype(f64).reshape(T, H, W), cache.float().numpy().astype(f64)
    far = base[3] + 5  # one key of a long sequence stands out
    cache[far] *= 6
    cv[far] *= 6
    dev = lambda a: torch.from_numpy(a).to(cuda)
    for sink in (None, rng.normal(2, 2, H).astype(np.float32)):
        want = attend(qv, cv, rank, base, last, W ** -0.5, None if sink is None else sink.astype(f64))
        for most in (701, part):  # (what sizes the split of the keys)
            got = ops.latent_attention(q.to(cuda), cache.to(cuda), dev(base), dev(last), H, rank, W ** -0.5, None if sink is None else dev(sink), most, False)
            got = got.float().cpu().numpy().reshape(T, H, rank)
            err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max(axis=(1, 2))
            assert err.max() < (2e-5 if dtype == torch.float32 else 0.012), err


@pytest.mark.parametrize("H,rank,rot", SIZES)
@pytest.mark.parametrize("first,T", [(0, 1), (0, 70), (130, 2), (61, 200)])
def test_a_chunk_of_a_prompt(cuda, H, rank, rot, first, T):
    rng = np.random.default_rng(2)
    W = rank + rot
    dev = lambda a: torch.from_numpy(a).to(cuda)
    for dtype in (torch.bfloat16, torch.float32):
        cache, q = draw(rng, 300, W, dtype=dtype), draw(rng, T, H * W, dtype=dtype)
        last = np.arange(first, first + T, dtype=np.int32)
        sink = rng.normal(1, 1, H).astype(np.float32)
        want = attend(q.float().numpy().astype(f64).reshape(T, H, W), cache.float().numpy().astype(f64), rank, np.zeros(T, int), last, 0.2, sink.astype(f64))
        got = ops.latent_attention(q.to(cuda), cache.to(cuda), None, dev(last), H, rank, 0.2, dev(sink), 300, True).float().cpu().numpy().reshape(T, H, rank)
        err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max(axis=(1, 2))
        assert err.max() < (2e-5 if dtype == torch.float32 else 0.012), (dtype, err.max(), err.argmax())


def test_scores_that_keep_growing_move_the_reference_maximum(cuda):
    # each tile of keys scores far above the one before, so the sums are rescaled again and again; and the other way round
    H, rank, rot, keys = 6, 128, 64, 512
    W = rank + rot
    for step in (1.0, -1.0):
        cache = torch.zeros(keys, W)
        cache[:, 0] = torch.from_numpy(1.0 + (np.arange(keys) // 16)[::int(step)].copy())
        cache[:, 1:] = torch.randn(keys, W - 1, generator=torch.Generator().manual_seed(3)) * 0.1
        q = torch.zeros(1, H, W)
        q[:, :, 0] = torch.linspace(0.25, 4, H)
        q, cache = q.bfloat16().reshape(1, H * W), cache.bfloat16()
        last = np.array([keys - 1], np.int32)
        want = attend(q.float().numpy().astype(f64).reshape(1, H, W), cache.float().numpy().astype(f64), rank, [0], last, 1.0, None)
        zero = torch.zeros(1, dtype=torch.int32, device=cuda)
        got = ops.latent_attention(q.to(cuda), cache.to(cuda), zero, torch.from_numpy(last).to(cuda), H, rank, 1.0, None, 64, False)  # (one CTA walks all the keys)
        got = got.float().cpu().numpy().reshape(1, H, rank)
        assert np.abs(got - want).max() < 0.01 * np.abs(want).max()


@pytest.mark.parametrize("q_rank,kv_rank,rot,dims", [(72, 96, 40, 40), (24, 40, 8, 4), (0, 64, 16, 16), (300, 33, 6, 2)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_latent_put_and_rotation(cuda, q_rank, kv_rank, rot, dims, dtype):
    from ferrite_b200 import mixers
    from ferrite_b200.tensor import Runtime
    from types import SimpleNamespace as NS
    rng, rt = np.random.default_rng(4), Runtime(0)
    T, eps = 6, 1e-3
    scaling = dict(factor=3.0, original=512, fast=16.0, slow=2.0)
    spec = dict(base=700.0, dims=dims, scaling=scaling if dims > 2 else None)
    freq, n, mag = mixers.rotation(rt, NS(base=700.0, dims=dims, scaling=NS(**scaling) if dims > 2 else None))
    down = draw(rng, T, q_rank + kv_rank + rot + 3, dtype=torch.float32)
    qn, kn = draw(rng, q_rank or 1, dtype=torch.float32), draw(rng, kv_rank, dtype=torch.float32)
    places, rows = np.array([0, 1, 2, 900, 5, 77], np.int32), np.array([4, 0, 9, 2, -1, 12], np.int32)
    cache = torch.full((10, kv_rank + rot), 3.0, dtype=dtype, device=cuda)
    q_out = torch.empty(T, q_rank, dtype=dtype, device=cuda) if q_rank else None
    dev = lambda a: torch.from_numpy(a).to(cuda)
    ops.latent_put(down.to(cuda), q_rank, kv_rank, rot, dims, qn.to(cuda) if q_rank else None, kn.to(cuda), eps, freq, mag, dev(places), dev(rows), cache, q_out)
    x = down.numpy().astype(f64)
    tol = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=8e-3, atol=8e-3)
    if q_rank:
        np.testing.assert_allclose(q_out.float().cpu().numpy(), oracle.rms(x[:, :q_rank], qn.numpy(), eps), **tol)
    part = x[:, q_rank + kv_rank:q_rank + kv_rank + rot]
    want = np.concatenate([oracle.rms(x[:, q_rank:q_rank + kv_rank], kn.numpy(), eps), oracle.rotate(part, places, spec)], 1)
    got = cache.float().cpu().numpy()
    for t, r in enumerate(rows):
        if 0 <= r < 10:
            np.testing.assert_allclose(got[r], want[t], **tol)
    assert (got[[1, 3, 5, 6, 7, 8]] == 3).all(), "rows that no token takes, and no row outside"
    heads = draw(rng, T, 5 * rot, dtype=dtype)
    out = torch.empty(T, 5 * (rot + 2), dtype=dtype, device=cuda)
    view = out.view(T, 5, rot + 2).permute(1, 0, 2)[:, :, 1:1 + rot] if dtype == torch.float32 else out.view(T, 5, rot + 2).permute(1, 0, 2)[:, :, :rot]
    ops.rotate_pairs(heads.to(cuda).view(T, 5, rot).permute(1, 0, 2), (freq, n, mag), dev(places), view)
    np.testing.assert_allclose(view.permute(1, 0, 2).float().cpu().numpy(), oracle.rotate(heads.float().numpy().astype(f64).reshape(T, 5, rot), places, spec), **tol)


DECAYS = [0.2, 0.61, 0.9, 0.97, 1.0, 0.999]


@pytest.mark.parametrize("H,dim,vdim", [(5, 32, 96), (2, 16, 48), (3, 128, 128), (1, 64, 32), (4, 20, 33), (2, 96, 256)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_decay_scan(cuda, H, dim, vdim, dtype):
    # a prompt in portions (down to one token), then one more token beside another sequence and a slot without a token;
    # the state that a slot held before is not seen by a sequence that starts in it
    rng = np.random.default_rng(5)
    cuts = [0, 2, 3, 67, 195, 330]
    T, decay = cuts[-1], np.array(DECAYS[:H], np.float32)
    n = H * (2 * dim + vdim)
    x = draw(rng, T + 1, n + 8, dtype=dtype, scale=0.6)
    xv = x.float().numpy().astype(f64)
    split = lambda v: (v[:, :H * dim].reshape(-1, H, dim), v[:, H * dim:2 * H * dim].reshape(-1, H, dim), v[:, 2 * H * dim:n].reshape(-1, H, vdim))
    state_want = np.zeros((H, dim, vdim))
    want = oracle.recurrence(*split(xv), decay.astype(f64), state_want)
    state = torch.randn(3, H * dim, vdim, device=cuda)
    left = state[2].clone()
    xd, dd = x.to(cuda), torch.from_numpy(decay).to(cuda)
    out = torch.empty(T + 1, H * vdim, device=cuda)
    place = lambda a, b: torch.arange(a, b, dtype=torch.int32, device=cuda)
    for a, b in zip(cuts, cuts[1:]):
        ops.decay_scan(xd[a:b], H, dim, vdim, dd, place(a, b), -1, state[1:2], out[a:b])
    three = torch.stack([xd[0], xd[T], xd[7]])
    three_out = torch.empty(3, H * vdim, device=cuda)
    ops.decay_scan(three, H, dim, vdim, dd, torch.tensor([0, T, 999], dtype=torch.int32, device=cuda), 999, state, three_out)
    out[T] = three_out[1]
    got = out.cpu().numpy().reshape(T + 1, H, vdim)
    err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max()
    assert err.max() < 3e-5, (err.max(), err.argmax())
    serr = np.abs(state[1].cpu().numpy().reshape(H, dim, vdim) - state_want).max(axis=(1, 2)) / np.abs(state_want).max(axis=(1, 2))
    assert serr.max() < 3e-5, serr
    np.testing.assert_allclose(three_out[0].cpu().numpy().reshape(H, vdim), want[0], rtol=1e-4, atol=1e-4 * np.abs(want[0]).max())
    assert torch.equal(state[2], left) and not three_out[2].any(), "a slot without a token keeps its state"


@pytest.mark.parametrize("cols,skip", [(333, 7), (96, 8), (2048, 0), (6000, 4), (5001, 3)])
def test_gated_rmsnorm(cuda, cols, skip):
    rng = np.random.default_rng(6)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 8e-3)):
        x, g, w = draw(rng, 5, cols, dtype=torch.float32), draw(rng, 5, cols + skip, dtype=dtype), draw(rng, cols, dtype=torch.float32)
        out = torch.empty(5, cols, dtype=dtype, device=cuda)
        ops.gated_rmsnorm(x.to(cuda), g.to(cuda)[:, skip:], w.to(cuda), 1e-4, out)
        want = oracle.rms(x.numpy().astype(f64), w.numpy(), 1e-4) * oracle.sigmoid(g.float().numpy().astype(f64)[:, skip:])
        np.testing.assert_allclose(out.float().cpu().numpy(), want, rtol=tol, atol=tol)
