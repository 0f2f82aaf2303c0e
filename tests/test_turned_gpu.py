"""The kernels of turned heads, windows, capped scores and corrected-score mixtures, each alone, against plain numpy: attention over
heads and over latents within a window, the projection's convolution, norms, turn and cache rows, queries taken apart and turned,
the GELU-gated matmul, routes with identity experts, the layer's end."""
from types import SimpleNamespace as NS

import numpy as np
import pytest

from conftest import to_numpy
from oracle import vunadra as oracle
from test_heads_gpu import Device, close, rounded

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def torch(cuda):
    import torch
    return torch


@pytest.fixture(scope="module")
def rt(cuda):
    from ferrite_b200.tensor import Runtime
    return Runtime(0)


def heads_case(torch, shape, bf16, places, window, cap, rng, seqs=None, plant=None, scale=None):
    from ferrite_b200 import ops
    (H, G, dim, vdim), T, n = shape, len(places), max(places) + 1
    on, S, part = Device(torch, bf16), seqs or 1, n + 5
    q, cache = rounded(rng.normal(0, 1, (T, H, dim)), bf16), rounded(rng.normal(0, 1, (G, S * part, dim + vdim)), bf16)
    if plant:
        plant(q, cache, part)
        q, cache = rounded(q, bf16), rounded(cache, bf16)
    scale = scale or 1.3 / np.sqrt(dim)
    base = [u * part for u in range(T)]
    got = ops.heads_attention(on(q.reshape(T, H * dim)), on(cache), on.i32(base) if seqs else None, on.i32(places), H, vdim, scale, n, not seqs, window=window or 0, softcap=cap or 0.0)
    want = np.zeros((T, H, vdim))
    for t, p in enumerate(places):
        rows = cache[:, base[t] if seqs else 0:][:, :p + 1].transpose(1, 0, 2)
        want[t] = oracle.attend(q[t:t + 1], rows[..., :dim], rows[..., dim:], [p], scale, window, cap)[0]
    return to_numpy(got), want.reshape(T, H * vdim)


# tensor-core sizes and others; window sizes at, below and above the tiles of 64 keys and of 1
@pytest.mark.parametrize("shape,bf16", [((8, 1, 40, 40), True), ((6, 2, 72, 24), True), ((2, 2, 256, 256), True), ((12, 4, 64, 64), False), ((3, 1, 9, 7), True), ((3, 3, 33, 65), False)])
def test_windows_and_capped_scores(torch, shape, bf16):
    rng = np.random.default_rng(0)
    for first, T, window, cap in ((0, 150, 48, 3.0), (0, 70, 64, None), (37, 70, 65, 2.0), (130, 33, None, 1.5), (158, 2, 63, None), (79, 3, 1, 5.0), (600, 20, 129, 4.0)):
        got, want = heads_case(torch, shape, bf16, list(range(first, first + T)), window, cap, rng)
        close(got, want, bf16, (first, T, window, cap))
    for places, window, cap in (([0, 1, 63, 64, 65, 127, 128, 300], 64, 3.0), ([79, 5, 160], 80, None), ([900, 3], None, 2.0), ([700], 1000, None), ([800, 40, 0], 300, 4.0), ([30, 31], 1, 1.0)):
        got, want = heads_case(torch, shape, bf16, places, window, cap, rng, seqs=len(places))
        close(got, want, bf16, (places, window, cap))


# prompts for the tcgen05 kernel: one group of pairs a CTA and two
@pytest.mark.parametrize("shape", [(64, 32, 80, 48), (40, 40, 64, 64), (37, 37, 256, 128), (74, 74, 8, 8), (160, 20, 128, 128)])
def test_windows_and_capped_scores_of_a_long_prompt(torch, shape):
    rng = np.random.default_rng(1)
    for first, T, window, cap in ((0, 200, 64, None), (37, 230, 97, 3.0), (300, 200, None, 1.5)):
        got, want = heads_case(torch, shape, True, list(range(first, first + T)), window, cap, rng)
        close(got, want, True, (first, T, window, cap))


def test_large_scores_stand_at_the_cap(torch):
    def plant(q, cache, part):  # scores of hundreds, both signs
        q *= 12
    for shape, T in (((4, 2, 64, 32), 30), ((74, 74, 64, 32), 200)):
        got, want = heads_case(torch, shape, True, list(range(T)), None, 6.0, np.random.default_rng(2), plant=plant, scale=1.0)
        close(got, want, True)


@pytest.mark.parametrize("kind,shape", [("prompt", (4, 2, 64, 32)), ("decode", (4, 2, 64, 32)), ("long prompt", (74, 74, 64, 32)), ("plain", (4, 2, 9, 7))])
@pytest.mark.parametrize("window", [40, 64])
def test_a_key_at_the_edge_of_a_window(torch, kind, shape, window):
    # one key scored far above all others: decides for tokens up to window - 1 past it, and is unseen from there on
    rng, key, dim = np.random.default_rng(3), 83, shape[2]
    places = list(range(key + window - 6, key + window + 6))

    def plant(q, cache, part):
        q[:] = q[:1, :1]
        for u in range(len(places) if kind == "decode" else 1):
            cache[:, u * part + key, :dim] = q[0, 0] * (2 if dim > 9 else 8)
            cache[:, u * part + key, dim:] = 8
    got, want = heads_case(torch, shape, kind != "plain", places, window, None, rng, seqs=len(places) if kind == "decode" else None, plant=plant)
    close(got, want, True)
    assert [bool(np.abs(row - 8).max() < 0.2) for row in got] == [p - key < window for p in places]


@pytest.mark.parametrize("H,rank,rot", [(12, 128, 48), (3, 64, 16), (16, 512, 64), (70, 96, 24), (5, 33, 7)])
@pytest.mark.parametrize("bf16", [True, False])
def test_windows_over_latents(torch, H, rank, rot, bf16):
    from ferrite_b200 import ops
    rng, on, W, part = np.random.default_rng(4), Device(torch, bf16), rank + rot, 700
    for places, chunk, window in (([0, 47, 48, 63, 64, 65, 650], False, 48), ([690, 31, 32, 33], False, 600), ([100, 3], False, 1), (list(range(90)), True, 33), (list(range(61, 200)), True, 64), (list(range(400, 402)), True, 300)):
        T = len(places)
        cache, q = rounded(rng.normal(0, 1, (part if chunk else T * part, W)), bf16), rounded(rng.normal(0, 1, (T, H, W)), bf16)
        base = [0] * T if chunk else [u * part for u in range(T)]
        for t, p in enumerate(places):  # the first key that is seen stands out, the one before it more so
            for back, much in ((window - 1, 1.5), (window, 4)):
                if p >= back and t == T - 1:
                    cache[base[t] + p - back] = rounded(q[t, 0] * much, bf16)
        got = ops.latent_attention(on(q.reshape(T, H * W)), on(cache), None if chunk else on.i32(base), on.i32(places), H, rank, 1.5 * W ** -0.5, None, part, chunk, window=window)
        for t, p in enumerate(places):
            rows = cache[base[t]:base[t] + p + 1, None]
            want = oracle.attend(q[t:t + 1], rows, rows[..., :rank], [p], 1.5 * W ** -0.5, window)
            close(to_numpy(got)[t], want.reshape(-1), bf16, (places[:3], window, t))


ROT = dict(base=700.0, scaling=dict(factor=3.0, original=512, fast=16.0, slow=2.0))


def rotation(rt, dims):
    from ferrite_b200 import mixers
    return mixers.rotation(rt, NS(base=ROT["base"], dims=dims, scaling=NS(**ROT["scaling"]))), dict(ROT, dims=dims)


# heads, key heads, key and value columns, turned columns, taps (0: no convolution), norms, keys that are the values, biases
@pytest.mark.parametrize("H,G,dim,vdim,dims,taps,norm,same,bias", [(12, 3, 40, 24, 40, 3, None, False, False), (4, 4, 64, 64, 20, 4, "heads", False, True), (6, 2, 72, 72, 72, 0, "all", True, True), (3, 1, 9, 9, 4, 2, "all", True, True),
                                                                   (3, 1, 7, 5, 0, 5, None, False, False), (40, 8, 128, 128, 128, 0, "all", False, True), (5, 5, 16, 8, 16, 1, None, False, True), (2, 1, 130, 260, 2, 3, "heads", False, False)])
@pytest.mark.parametrize("source,bf16", [("fp32", True), ("fp32", False), ("bf16", True)])
def test_convolution_norms_turn_and_cache_rows(torch, rt, H, G, dim, vdim, dims, taps, norm, same, bias, source, bf16):
    from ferrite_b200 import ops
    rng, on, src = np.random.default_rng(5), Device(torch, bf16), Device(torch, source == "bf16")
    wide = (H + G) * dim + (0 if same else G * vdim)
    f32 = lambda a: np.float64(np.float32(a))
    b = f32(rng.normal(0, 1, wide)) if bias else None
    qn, kn = (f32(rng.normal(1, 0.3, n * dim if norm == "all" else dim)) for n in (H, G))
    conv = f32(rng.normal(0, 0.8, (taps, wide))) if taps else None
    turn, spec = rotation(rt, dims) if dims else (None, None)
    n, slots, part = 23, 3, 40
    x = rounded(rng.normal(0, 1, (n + 1, wide + 4)), source == "bf16")
    y = x[:, :wide] + (b if bias else 0)
    u = oracle.convolved(y, conv.T, np.zeros((taps - 1, wide)))[0] if taps else y
    q, k = u[:, :H * dim], u[:, H * dim:(H + G) * dim]
    v = (k if same else u[:, (H + G) * dim:]).reshape(-1, G, vdim)
    if norm == "all":
        q, k = oracle.rms(q, qn, 1e-2), oracle.rms(k, kn, 1e-2)
    q, k = q.reshape(-1, H, dim), k.reshape(-1, G, dim)
    if norm == "heads":
        q, k = oracle.rms(q, qn, 1e-2), oracle.rms(k, kn, 1e-2)
    if dims:
        q, k = oracle.rotate(q, range(n + 1), spec), oracle.rotate(k, range(n + 1), spec)
    tol = 6e-3 if bf16 else 1e-5
    for cuts in ([n], [1] * 6 + [n - 6], [2, 2, 1, n - 5], [n - 1, 1]):
        cache = on(np.full((G, slots * part, dim + vdim), 7.0))
        state = torch.randn(slots, max(taps - 1, 1), wide, device="cuda")
        left, qs, at = state.clone(), [], 0
        kw = dict(bias=on.f32(b) if bias else None, q_norm=on.f32(qn) if norm else None, k_norm=on.f32(kn) if norm else None, eps=1e-2, norm_all=norm == "all", keys_are_values=same, rotation=turn,
                  conv=on.f32(conv) if taps else None)
        for m in cuts:  # slot 1's prompt in portions
            out = on(np.zeros((m, H * dim)))
            places = np.arange(at, at + m)
            ops.heads_put(src(x[at:at + m]), H, G, dim, vdim, on.i32(part + places), cache, out, places=on.i32(places), state=state[1:2] if taps else None, **kw)
            qs.append(to_numpy(out))
            at += m
        # then a token of each slot: one that begins in a used slot, slot 1's next, none
        out = on(np.zeros((3, H * dim)))
        ops.heads_put(src(x[[0, n, 5]]), H, G, dim, vdim, on.i32([0, part + n, -1]), cache, out, places=on.i32([0, n, part - 1]), state=state if taps else None, dead=part - 1, **kw)
        np.testing.assert_allclose(np.concatenate(qs + [to_numpy(out)[1:2], to_numpy(out)[:1]]), np.concatenate([q, q[:1]]).reshape(n + 2, -1), rtol=tol, atol=tol * 3)
        want = np.full((G, slots * part, dim + vdim), 7.0)
        want[:, part:part + n + 1, :dim], want[:, part:part + n + 1, dim:] = k.transpose(1, 0, 2), v.transpose(1, 0, 2)
        want[:, 0, :dim], want[:, 0, dim:] = k[0], v[0]
        np.testing.assert_allclose(to_numpy(cache), want, rtol=tol, atol=tol * 3)
        if taps > 1:
            np.testing.assert_allclose(to_numpy(state)[1], y[n + 2 - taps:n + 1], rtol=1e-6, atol=1e-6)
            np.testing.assert_allclose(to_numpy(state)[0], np.concatenate([np.zeros((taps - 2, wide)), y[:1]]), rtol=1e-6, atol=1e-6)
            assert torch.equal(state[2], left[2]), "a slot without a token keeps its state"


@pytest.mark.parametrize("H,dim,rank,rot,dims", [(5, 24, 40, 16, 16), (3, 11, 33, 7, 4), (32, 128, 512, 64, 64)])
@pytest.mark.parametrize("bf16", [True, False])
def test_queries_taken_apart_and_turned(torch, rt, H, dim, rank, rot, dims, bf16):
    from ferrite_b200 import ops
    rng, on, T = np.random.default_rng(6), Device(torch, bf16), 6
    (freq, n, mag), spec = rotation(rt, dims)
    x, kn = (np.float64(np.float32(rng.normal(0, 1, s))) for s in ((T, H * (dim + rot) + rank + rot + 3), rank))
    places, rows = [0, 1, 900, 5, 77, 12], [4, 0, 9, -1, 10, 2]
    cache, plain, query = on(np.full((10, rank + rot), 3.0)), on(np.zeros((T, H * dim))), on(np.full((T, H * (rank + rot)), 5.0))
    turned = query.view(T, H, rank + rot).permute(1, 0, 2)[:, :, rank:]
    ops.latent_put(on.f32(x), 0, rank, rot, dims, None, on.f32(kn), 1e-3, freq, mag, on.i32(places), on.i32(rows), cache, plain, H, dim, turned)
    q = x[:, :H * (dim + rot)].reshape(T, H, dim + rot)
    tol = dict(rtol=8e-3, atol=8e-3) if bf16 else dict(rtol=2e-5, atol=2e-5)
    np.testing.assert_allclose(to_numpy(plain), q[..., :dim].reshape(T, -1), **tol)
    got = to_numpy(query).reshape(T, H, rank + rot)
    np.testing.assert_allclose(got[..., rank:], oracle.rotate(q[..., dim:], places, spec), **tol)
    assert (got[..., :rank] == 5).all()
    down = x[:, H * (dim + rot):]
    want = np.concatenate([oracle.rms(down[:, :rank], kn, 1e-3), oracle.rotate(down[:, None, rank:rank + rot], places, spec)[:, 0]], 1)
    for t, r in enumerate(rows):
        if 0 <= r < 10:
            np.testing.assert_allclose(to_numpy(cache)[r], want[t], **tol)
    assert (to_numpy(cache)[[1, 3, 5, 6, 7, 8]] == 3).all()


@pytest.mark.parametrize("M,K,N", [(1, 256, 64), (20, 96, 416), (130, 1024, 1056), (300, 264, 160), (4, 4096, 512), (7, 60, 26)])
@pytest.mark.parametrize("bias", [True, False])
def test_gelu_gated_matmul(torch, rt, M, K, N, bias):
    from ferrite_b200.tensor import Tensor
    rng = np.random.default_rng(7)
    for dtype, tol in (("bf16", 8e-3), ("fp32", 3e-6)):
        bf16 = dtype == "bf16"
        x, w, b = rounded(rng.normal(0, 1, (M, K)), bf16), rounded(rng.normal(0, 2 * K ** -0.5, (N, K)), bf16), np.float64(np.float32(rng.normal(0, 1, (1, N))))
        before = rt.launches
        got = Tensor.of(rt, x, dtype).matmul(Tensor.of(rt, w, dtype).T, dtype="fp32").gelu_gated(Tensor.of(rt, b, "fp32") if bias else None, dtype).realize()
        fused = "dense geglu" in [n for n, _ in rt.profile(before)]
        assert got.dtype == dtype and (fused or len(rt.names) >= 4096) == (bf16 and N % 32 == 0 and K % 8 == 0) or len(rt.names) >= 4096
        y = x @ w.T + (b if bias else 0)
        want = oracle.gelu(y[:, :N // 2]) * y[:, N // 2:]
        assert np.abs(got.numpy()[0] - want).max() <= tol * np.abs(want).max()


@pytest.mark.parametrize("T,n,identity,k", [(1, 7, 2, 2), (7, 11, 3, 11), (33, 128, 8, 8), (64, 6, 5, 3), (65, 130, 30, 3), (200, 8, 0, 2), (700, 40, 4, 32), (130, 9, 8, 1), (1500, 300, 20, 6)])
def test_scored_routes_with_identity_experts(torch, T, n, identity, k):
    from ferrite_b200 import ops
    rng, on, real = np.random.default_rng(8), Device(torch, False), n - identity
    z = np.argsort(rng.random((T, n)), 1) * (9.0 / n) + rng.normal(0, 0.2 / n, (T, n))  # (no close calls)
    c = np.zeros(n)
    c[rng.integers(n)], c[rng.integers(n)] = 2.0, -2.0
    z, c = np.float64(np.float32(z)), np.float64(c)
    r = ops.route(on(z), n, k, on(c), True, identity, 1.7)
    picks, weight = oracle.route(z, dict(router=np.eye(n), correction=c), "", dict(top=k, scale=1.7))
    assert np.array_equal(to_numpy(r.ids), picks)
    np.testing.assert_allclose(to_numpy(r.weights), weight, rtol=2e-5, atol=1e-7)
    live, experts, slots = int(to_numpy(r.live)[0]), to_numpy(r.tile_expert)[:, 0], to_numpy(r.slots)
    count = np.bincount(picks.reshape(-1), minlength=n)[:real]
    assert live == ((count > 0) if r.shared else -(-count // r.tile)).sum() <= r.tiles and (experts[live:] == real).all()
    assert ((slots < 0) == (picks >= real)).all() and np.array_equal(experts[slots[slots >= 0] // r.tile], picks[picks < real])
    assert r.shared or len(set(slots[slots >= 0].tolist())) == (slots >= 0).sum()


@pytest.mark.parametrize("T,n,identity,k,K,m,bf16", [(1, 6, 2, 2, 64, 32, True), (32, 10, 1, 3, 320, 80, True), (300, 11, 4, 4, 192, 48, True), (30, 5, 2, 3, 60, 13, True), (100, 5, 2, 3, 60, 13, False), (9, 1, 3, 2, 64, 32, True),
                                                     (80, 1, 3, 2, 64, 32, True)])
def test_clamped_experts_and_their_sum(torch, rt, T, n, identity, k, K, m, bf16):
    from ferrite_b200.tensor import Tensor
    rng, limit = np.random.default_rng(9), 0.9
    kind = "bf16" if bf16 else "fp32"
    w = {f"e{e}.{name}": rounded(rng.normal(0, 1.5 * shape[1] ** -0.5, shape), bf16) for e in range(n) for name, shape in (("gate", (m, K)), ("up", (m, K)), ("down", (K, m)))}
    h, x = rounded(rng.normal(0, 1, (T, K)), bf16), np.float64(np.float32(rng.normal(0, 1, (T, K))))
    z = np.argsort(rng.random((T, n + identity)), 1) * (5.0 / (n + identity))
    if n == 1 and T == 9:
        z[:, 0] = -9  # nobody takes an expert with rows
    w |= dict(router=np.eye(n + identity), correction=np.zeros(n + identity))
    stack = lambda f: Tensor.of(rt, np.stack([f(e) for e in range(n)]), kind).T
    routes = Tensor.of(rt, z, "fp32").route(n + identity, k, None, True, identity, 1.3)
    hd = Tensor.of(rt, h, kind)
    rows = hd.experts(routes, stack(lambda e: np.concatenate([w[f"e{e}.gate"], w[f"e{e}.up"]])), stack(lambda e: w[f"e{e}.down"]), (limit, oracle.SLOPE))
    got, _ = Tensor.of(rt, x, "fp32").add_norm(Tensor.of(rt, np.ones((1, K)), "fp32"), 1e-3, dtype=kind, experts=(rows, routes), own=hd)
    picks, weight = oracle.route(np.float64(np.float32(z)), w, "", dict(top=k, scale=1.3))
    want = x.copy()
    for t in range(T):
        for e, s in zip(picks[t], weight[t]):
            want[t] += s * (oracle.expert(h[t:t + 1], w, f"e{e}.", limit)[0] if e < n else h[t])
    assert np.abs(got.numpy()[0] - want).max() < (2e-2 if bf16 else 5e-6) * np.abs(want).max()


@pytest.mark.parametrize("cols,source,bf16", [(288, "bf16", True), (260, "fp32", True), (61, "fp32", False), (61, "bf16", True), (4096, "fp32", True), (9000, "fp32", False)])
def test_biases_and_rows_as_they_are_at_the_end_of_a_layer(torch, cols, source, bf16):
    from ferrite_b200 import ops
    rng, on, src, T = np.random.default_rng(10), Device(torch, bf16), Device(torch, source == "bf16"), 7
    x, b, w = (np.float64(np.float32(rng.normal(0, 1, s))) for s in ((T, cols), cols, cols))
    y = rounded(rng.normal(0, 1, (T, cols)), source == "bf16")
    tol = 6e-3 if bf16 else 1e-5
    for mixer, norm in ((1, 1), (0, 1), (1, 0), (0, 0)):
        wide = on(np.full((T, 2 * cols), 9.0))  # (the second result beside another's columns)
        out, h = on.f32(np.zeros((T, cols))), wide[:, cols:] if cols % 2 else wide[:, :cols]
        ops.add_norm(on.f32(x), out, src(y) if mixer else None, None, w=on.f32(w) if norm else None, eps=1e-3, h=h, mixer_bias=on.f32(b))
        want = x + mixer * y + b
        np.testing.assert_allclose(to_numpy(out), want, rtol=1e-5, atol=2e-5)
        np.testing.assert_allclose(to_numpy(h), oracle.rms(want, w, 1e-3) if norm else want, rtol=tol, atol=tol)
        assert (to_numpy(wide[:, :cols] if cols % 2 else wide[:, cols:]) == 9).all()


def test_scaled_embedding(torch):
    from ferrite_b200 import ops
    rng, on = np.random.default_rng(11), Device(torch, True)
    a = rounded(rng.normal(0, 1, (20, 61)), True)
    out = ops.embed(on(a), on.i32([3, 0, 19]), None, None, on.f32(np.zeros((3, 61))), 0.3)
    np.testing.assert_allclose(to_numpy(out), a[[3, 0, 19]] * np.float32(0.3), rtol=1e-6)
