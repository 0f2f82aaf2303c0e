"""The kernels of state spaces, gated recurrences, attention weighted by sigmoids, squared-ReLU mixtures and gated, normed layer ends,
each alone, against plain numpy."""
from types import SimpleNamespace as NS

import numpy as np
import pytest

from conftest import to_numpy
from oracle import ronavik as oracle
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


def f32(a):
    return np.asarray(a, np.float32).astype(np.float64)


# how a sequence of 331 tokens is cut, down to one token; the last one goes beside other sequences
CUTS = [0, 2, 3, 66, 195, 211, 330]


def in_portions(torch, on, T, run, state, mine=1):
    """run(rows, places, dead, state, out rows) over slot `mine` of a state for three in portions, then over a token of each: one that begins in a used slot, `mine`'s
    next, none."""
    for a, b in zip(CUTS, CUTS[1:]):
        run(slice(a, b), on.i32(np.arange(a, b)), -1, [s[mine:mine + 1] for s in state], slice(a, b))
    run([0, T, 7], on.i32([0, T, 999]), 999, state, None)


# ---- the state space

@pytest.mark.parametrize("H,G,dim,vdim", [(5, 5, 32, 96), (6, 2, 16, 48), (4, 1, 128, 64), (3, 3, 64, 32), (4, 2, 20, 33), (2, 1, 96, 256), (8, 4, 1, 1), (3, 1, 240, 40), (2, 2, 300, 24), (6, 3, 48, 72), (2, 1, 128, 136), (9, 3, 112, 8), (2, 2, 96, 64)])
@pytest.mark.parametrize("bf16", [True, False])
def test_selective_scan(torch, H, G, dim, vdim, bf16):
    from ferrite_b200 import ops
    rng, on, T = np.random.default_rng(0), Device(torch, bf16), CUTS[-1]
    n = H * vdim + 2 * G * dim
    x, dt = rounded(rng.normal(0, 0.6, (T + 1, n + 8)), bf16), f32(rng.normal(-1, 1.5, (T + 1, H + 3)))
    dt[100], dt[160] = 60, -60  # a token that all but replaces the state, one that all but leaves it
    bias, a_log, skip = (f32(rng.normal(m, 1, H)) for m in (-0.5, -1.5, 1))
    # (a slow head: hundreds of tokens count)
    a_log[0] = -6
    parts = lambda v: (v[:, :H * vdim].reshape(-1, H, vdim), v[:, H * vdim:H * vdim + G * dim].reshape(-1, G, dim), v[:, H * vdim + G * dim:n].reshape(-1, G, dim))
    step = oracle.softplus(dt[:, :H] + bias)
    want, last = oracle.state_space(*parts(x), step, a_log, np.zeros((H, dim, vdim)))
    want += skip[:, None] * parts(x)[0]
    state = torch.randn(3, H * dim, vdim, device="cuda")
    left, out, three = state[2].clone(), torch.empty(T, H * vdim, device="cuda"), torch.empty(3, H * vdim, device="cuda")
    xd, dd = on(x), on.f32(dt)

    def run(rows, places, dead, s, to):
        ops.selective_scan(xd[rows], H, G, dim, vdim, dd[rows][:, :H], on.f32(bias), on.f32(a_log), on.f32(skip), places, dead, s[0] if isinstance(s, list) else s, three if to is None else out[to])
    in_portions(torch, on, T, run, [state])
    got = np.concatenate([to_numpy(out), to_numpy(three)[1:2]]).reshape(T + 1, H, vdim)
    for h in range(H):  # (each head by its own size)
        assert np.abs(got[:, h] - want[:, h]).max() < 5e-5 * np.abs(want[:, h]).max(), h
        assert np.abs(to_numpy(state)[1].reshape(H, dim, vdim)[h] - last[h]).max() < 5e-5 * np.abs(last[h]).max(), h
    np.testing.assert_allclose(to_numpy(three)[0].reshape(H, vdim), want[0], rtol=1e-4, atol=1e-4 * np.abs(want[0]).max())
    assert torch.equal(state[2], left) and not three[2].any(), "a slot without a token keeps its state"


def test_selective_scan_of_a_long_prompt_and_of_several(torch):
    # chunk after chunk, a state that lasts, and rows of another sequence right after a sequence's last
    from ferrite_b200 import ops
    rng, on, (H, G, dim, vdim) = np.random.default_rng(15), Device(torch, True), (4, 2, 64, 48)
    for sequences, T in ((1, 1500), (3, 200), (2, 129), (5, 65)):
        n = H * vdim + 2 * G * dim
        x, dt = rounded(rng.normal(0, 0.6, (sequences * T, n)), True), f32(rng.normal(-1, 1.5, (sequences * T, H)))
        bias, a_log, skip = f32(rng.normal(-3, 1, H)), f32([-7.0, -4, -1, 1]), f32(rng.normal(1, 1, H))
        state, out = torch.randn(sequences, H * dim, vdim, device="cuda"), torch.empty(sequences * T, H * vdim, device="cuda")
        before = to_numpy(state).reshape(sequences, H, dim, vdim)
        places = np.concatenate([np.arange(T) + 10 * (s == 1) for s in range(sequences)])  # (the second goes on, the others begin)
        ops.selective_scan(on(x), H, G, dim, vdim, on.f32(dt), on.f32(bias), on.f32(a_log), on.f32(skip), on.i32(places), -1, state, out)
        for s in range(sequences):
            v = x[s * T:(s + 1) * T]
            parts = v[:, :H * vdim].reshape(-1, H, vdim), v[:, H * vdim:H * vdim + G * dim].reshape(-1, G, dim), v[:, H * vdim + G * dim:].reshape(-1, G, dim)
            want, last = oracle.state_space(*parts, oracle.softplus(dt[s * T:(s + 1) * T] + bias), a_log, before[s] if s == 1 else np.zeros((H, dim, vdim)))
            want += skip[:, None] * parts[0]
            got = to_numpy(out)[s * T:(s + 1) * T].reshape(T, H, vdim)
            for h in range(H):
                assert np.abs(got[:, h] - want[:, h]).max() < 5e-5 * np.abs(want[:, h]).max(), (sequences, T, s, h)
                assert np.abs(to_numpy(state)[s].reshape(H, dim, vdim)[h] - last[h]).max() < 5e-5 * np.abs(last[h]).max(), (sequences, T, s, h)


@pytest.mark.parametrize("cols,parts,skip", [(333, 3, 7), (96, 8, 8), (2048, 1, 0), (6000, 1, 4), (6000, 4, 4), (5001, 1, 3), (64, 64, 4)])
@pytest.mark.parametrize("before", [True, False])
def test_gates_before_and_after_a_norm_in_parts(torch, cols, parts, skip, before):
    from ferrite_b200 import ops
    rng = np.random.default_rng(1)
    for gate, bf16, tol in ((False, False, 2e-5), (False, True, 8e-3), (True, True, 8e-3)):
        on, src = Device(torch, bf16), Device(torch, gate)
        x, g, w = f32(rng.normal(0, 1, (5, cols))), rounded(rng.normal(0, 1.5, (5, cols + skip)), gate), f32(rng.normal(1, 0.3, cols))
        x[:, :cols // parts] *= 7  # (the parts' own sizes differ)
        out = on(np.zeros((5, cols)))
        ops.gated_rmsnorm(on.f32(x), src(g)[:, skip:], on.f32(w), 1e-3, out, before, parts)
        g = g[:, skip:]
        y = (x * oracle.silu(g) if before else x).reshape(5, parts, -1)
        want = oracle.rms(y, 1.0, 1e-3).reshape(5, cols) * w * (1 if before else oracle.sigmoid(g))
        np.testing.assert_allclose(to_numpy(out), want, rtol=tol, atol=tol)


# ---- the short convolution

@pytest.mark.parametrize("cols,skip", [(96, 4), (61, 2), (1040, 0)])
@pytest.mark.parametrize("taps,silu,in_bias,bias", [(4, True, False, True), (4, False, True, True), (3, False, False, False), (2, True, True, False), (1, False, True, True), (7, True, False, True)])
def test_short_convolution(torch, cols, skip, taps, silu, in_bias, bias):
    from ferrite_b200 import ops
    rng, T = np.random.default_rng(2), CUTS[-1]
    w, b, ib = f32(rng.normal(0, 0.7, (taps, cols))), f32(rng.normal(0, 1, cols)), f32(rng.normal(0, 1, cols))
    for source, bf16 in ((False, True), (False, False), (True, True)):
        on, src = Device(torch, bf16), Device(torch, source)
        x = rounded(rng.normal(0, 1, (T + 1, cols + skip)), source)
        u = x[:, skip:] + (ib if in_bias else 0)
        want = oracle.short_convolution(u, {"c": w.T, "c.b": b if bias else 0.0}, "c", {})
        want = oracle.silu(want) if silu else want
        state = torch.randn(3, max(taps - 1, 1), cols, device="cuda")
        left, out, three, xd = state.clone(), on(np.zeros((T, cols))), on(np.zeros((3, cols))), src(x)

        def run(rows, places, dead, s, to):
            ops.short_conv(xd[rows][:, skip:], on.f32(w), three if to is None else out[to], places, dead, s[0] if isinstance(s, list) else s, on.f32(b) if bias else None, on.f32(ib) if in_bias else None, silu)
        in_portions(torch, on, T, run, [state])
        tol = 8e-3 if bf16 else 1e-5
        np.testing.assert_allclose(np.concatenate([to_numpy(out), to_numpy(three)[1:2]]), want, rtol=tol, atol=tol)
        np.testing.assert_allclose(to_numpy(three)[0], want[0], rtol=tol, atol=tol)
        if taps > 1:
            np.testing.assert_allclose(to_numpy(state)[1], u[T + 2 - taps:T + 1], rtol=1e-6, atol=1e-6)
            np.testing.assert_allclose(to_numpy(state)[0], np.concatenate([np.zeros((taps - 2, cols)), u[:1]]), rtol=1e-6, atol=1e-6)
        assert torch.equal(state[2], left[2]), "a slot without a token keeps its state"


# ---- the gated linear recurrence

@pytest.mark.parametrize("width,blocks,skip", [(96, 4, 4), (35, 5, 3), (1, 1, 0), (512, 2, 8), (1000, 1, 0)])
def test_gated_recurrence(torch, width, blocks, skip):
    from ferrite_b200 import ops
    rng, T, part = np.random.default_rng(3), CUTS[-1], width // blocks
    lam, y_bias = f32(rng.normal(-2, 3, width)), f32(rng.normal(0, 1, width))
    lam[0] = -16  # a column that hardly forgets
    gate_bias = f32(rng.normal(0, 1, (blocks, 2 * part)))
    for source, bf16 in ((False, True), (False, False), (True, True)):
        on, src = Device(torch, bf16), Device(torch, source)
        u, y = rounded(rng.normal(0, 1, (T + 1, width)), bf16), rounded(rng.normal(0, 1.5, (T + 1, width + skip)), source)
        gates = f32(rng.normal(0, 2, (T + 1, 2 * width)))
        r, i = (oracle.sigmoid((gates.reshape(-1, blocks, 2, part) + gate_bias.reshape(blocks, 2, part))[:, :, k].reshape(-1, width)) for k in (0, 1))
        s, last = oracle.recurrence(u, r, i, lam, np.zeros(width))
        want = 0.7 * s * oracle.gelu(y[:, skip:] + y_bias)
        state = torch.randn(3, 1, width, device="cuda")
        left, wide, three, ud, yd, gd = state.clone(), on(np.full((T, width + 8), 9.0)), on(np.zeros((3, width))), on(u), src(y), on.f32(gates)

        def run(rows, places, dead, st, to):
            ops.lru_scan(ud[rows], gd[rows], yd[rows][:, skip:], three if to is None else wide[to][:, 8:], on.f32(lam), -8.0, blocks, places, dead, st[0] if isinstance(st, list) else st, on.f32(gate_bias), on.f32(y_bias), 0.7)
        in_portions(torch, on, T, run, [state])
        tol = 8e-3 if bf16 else 2e-5
        got = np.concatenate([to_numpy(wide)[:, 8:], to_numpy(three)[1:2]])
        assert (np.abs(got - want) <= tol * np.abs(want) + (1e-5 * np.abs(s).max() if not bf16 else 1e-4)).all()
        np.testing.assert_allclose(to_numpy(state)[1, 0], last, rtol=2e-5, atol=2e-6)
        np.testing.assert_allclose(to_numpy(three)[0], want[0], rtol=tol, atol=1e-4)
        assert torch.equal(state[2], left[2]) and not three[2].any() and (to_numpy(wide)[:, :8] == 9).all()


# ---- attention whose weights are sigmoids

def sigmoid_case(torch, shape, bf16, places, rng, seqs=None, plant=None, scale=None, bias=None, padded=3):
    from ferrite_b200 import ops
    (H, G, dim, vdim), T, n = shape, len(places), max(places) + 1
    on, S, part = Device(torch, bf16), seqs or 1, n + 5
    q, cache = rounded(rng.normal(0, 1, (T, H, dim)), bf16), rounded(rng.normal(0, 1, (G, S * part, dim + vdim)), bf16)
    bias = f32(rng.normal(-2, 1.5, H) if bias is None else np.full(H, bias))
    if plant:
        plant(q, cache, part)
        q, cache = rounded(q, bf16), rounded(cache, bf16)
    scale = scale or 1.3 / np.sqrt(dim)
    base = [u * part for u in range(T)]
    wide = on(np.full((T, H * vdim + padded), 5.0))
    ops.heads_attention(on(q.reshape(T, H * dim)), on(cache), on.i32(base) if seqs else None, on.i32(places), H, vdim, scale, n, not seqs, key_bias=on.f32(bias), out_scale=0.7, out=wide[:, :H * vdim])
    assert (to_numpy(wide)[:, H * vdim:] == 5).all()
    want = np.zeros((T, H, vdim))
    for t, p in enumerate(places):
        rows = cache[:, base[t] if seqs else 0:][:, :p + 1].transpose(1, 0, 2)
        want[t] = 0.7 * oracle.attend(q[t:t + 1], rows[..., :dim], rows[..., dim:], [p], scale, bias)[0]
    return to_numpy(wide)[:, :H * vdim], want.reshape(T, H * vdim)


# every padded size of the tensor-core kernel, more query heads a key head than a tile has rows; odd sizes and fp32 for the general one
@pytest.mark.parametrize("shape,bf16", [((8, 1, 40, 40), True), ((6, 2, 72, 24), True), ((2, 2, 256, 256), True), ((40, 2, 136, 72), True), ((4, 2, 104, 208), True), ((12, 4, 64, 64), False), ((3, 1, 9, 7), True), ((3, 3, 33, 65), False), ((1, 1, 8, 300), True)])
def test_attention_by_sigmoids(torch, shape, bf16):
    rng = np.random.default_rng(4)
    for first, T in ((0, 150), (0, 1), (37, 70), (158, 2), (600, 20)):
        close(*sigmoid_case(torch, shape, bf16, list(range(first, first + T)), rng, padded=4 if T % 2 else 8), bf16, (first, T))
    for places in ([0, 1, 63, 64, 65, 127, 128, 300], [900, 3], [700], [0], [1500, 800, 40, 0]):
        close(*sigmoid_case(torch, shape, bf16, places, rng, seqs=len(places)), bf16, places)


# prompts for the tcgen05 kernel: one group of pairs a CTA and two, and values that take all of tensor memory
@pytest.mark.parametrize("shape", [(64, 32, 80, 48), (40, 40, 64, 64), (37, 37, 256, 128), (74, 74, 8, 8), (160, 20, 128, 128), (80, 20, 64, 256), (40, 40, 104, 208), (37, 37, 72, 136)])
def test_attention_by_sigmoids_of_a_long_prompt(torch, shape):
    rng = np.random.default_rng(5)
    for first, T, padded in ((0, 200, 0), (37, 230, 2), (300, 200, 1)):
        close(*sigmoid_case(torch, shape, True, list(range(first, first + T)), rng, padded=padded), True, (first, T))


# softmax prompts with wide values go the same way now
@pytest.mark.parametrize("shape", [(80, 20, 64, 256), (37, 37, 72, 136)])
def test_softmax_of_a_long_prompt_with_wide_values(torch, shape):
    from test_turned_gpu import heads_case
    rng = np.random.default_rng(6)
    for first, T, window, cap in ((0, 200, None, None), (37, 230, 97, 3.0)):
        close(*heads_case(torch, shape, True, list(range(first, first + T)), window, cap, rng), True, (first, T))


@pytest.mark.parametrize("kind,shape", [("prompt", (4, 2, 64, 32)), ("decode", (4, 2, 64, 32)), ("long prompt", (74, 74, 64, 32)), ("wide prompt", (74, 74, 64, 200)), ("plain", (4, 2, 9, 7))])
def test_one_far_key_among_many(torch, kind, shape):
    # all weights but that of one key are next to nothing: it is felt from its own place on, far past it, with the weight its score gives
    rng, dim = np.random.default_rng(7), shape[2]
    for key in (0, 63, 64, 150):
        places = sorted({max(key - 1, 0), key, key + 1, key + 63, key + 64, key + 300, 620}) if kind == "decode" else list(range(max(key - 3, 0), max(key - 3, 0) + 150))

        def plant(q, cache, part):
            q[:] = q[:1, :1]
            for u in range(len(places) if kind == "decode" else 1):
                cache[:, u * part + key, :dim] = q[0, 0] * (20 / (q[0, 0] ** 2).sum() / 0.3)
                cache[:, u * part + key, dim:] = 8
        got, want = sigmoid_case(torch, shape, kind != "plain", places, rng, seqs=len(places) if kind == "decode" else None, plant=plant, scale=0.3 if dim > 9 else 0.05, bias=-19.0 if dim > 9 else -6.0)
        close(got, want, True)
        if dim > 9:
            assert [bool(np.abs(row).max() > 2) for row in got] == [p >= key for p in places]


def test_large_scores_of_both_signs(torch):
    def plant(q, cache, part):
        q *= 40
    for shape, T, bf16 in (((4, 2, 64, 32), 30, True), ((74, 74, 64, 32), 200, True), ((4, 2, 64, 32), 30, False)):
        got, want = sigmoid_case(torch, shape, bf16, list(range(T)), np.random.default_rng(8), plant=plant, scale=1.0)
        close(got, want, True)
        assert np.isfinite(got).all()


@pytest.mark.parametrize("H,G,dim,vdim,dims", [(4, 2, 40, 24, 0), (12, 3, 128, 256, 0), (3, 1, 9, 7, 0), (3, 1, 300, 8, 0), (4, 2, 24, 24, 12)])
@pytest.mark.parametrize("coef,every", [(0.5, 8), (-0.2, 1), (1.3, 1000)])
def test_queries_by_the_temperature_of_their_place(torch, rt, H, G, dim, vdim, dims, coef, every):
    from ferrite_b200 import mixers, ops
    from oracle import vunadra
    rng = np.random.default_rng(9)
    places = [0, every - 1, every, every + 1, 7, 15, 16, 5000] if every > 1 else [0, 1, 2, 3, 7, 15, 16, 5000]
    T, wide = len(places), (H + G) * dim + G * vdim
    for bf16, tol in ((True, 8e-3), (False, 2e-5)):
        on = Device(torch, bf16)
        x, qn, kn = f32(rng.normal(0, 1, (T, wide + 4))), f32(rng.normal(1, 0.3, dim)), f32(rng.normal(1, 0.3, dim))
        cache, q_out = on(np.full((G, T + 2, dim + vdim), 3.0)), on(np.zeros((T, H * dim)))
        rot = NS(base=50.0, dims=dims, scaling=None)
        ops.heads_put(on.f32(x)[:, 4:], H, G, dim, vdim, on.i32(np.arange(T)), cache, q_out, q_norm=on.f32(qn), k_norm=on.f32(kn), eps=1e-3, places=on.i32(places), temperature=(coef, every),
                      rotation=mixers.rotation(rt, rot) if dims else None)
        x = x[:, 4:]
        q, k = (oracle.rms(x[:, a:b].reshape(T, -1, dim), n, 1e-3) for a, b, n in ((0, H * dim, qn), (H * dim, (H + G) * dim, kn)))
        if dims:
            q, k = (vunadra.rotate(v, places, dict(base=50.0, dims=dims)) for v in (q, k))
        q = q * np.array([oracle.temperature(p, dict(coef=coef, every=every)) for p in places])[:, None, None]
        np.testing.assert_allclose(to_numpy(q_out), q.reshape(T, -1), rtol=tol, atol=tol)
        np.testing.assert_allclose(to_numpy(cache)[:, :T, :dim], k.transpose(1, 0, 2), rtol=tol, atol=tol)
        np.testing.assert_allclose(to_numpy(cache)[:, :T, dim:], x[:, (H + G) * dim:].reshape(T, G, vdim).transpose(1, 0, 2), rtol=tol, atol=tol)


# ---- the mixture

@pytest.mark.parametrize("T,n,k", [(1, 7, 2), (7, 11, 11), (33, 128, 8), (64, 6, 1), (65, 130, 3), (200, 8, 2), (1500, 300, 6)])
@pytest.mark.parametrize("shares,correction", [(False, False), (True, True)])
def test_sigmoid_routes(torch, T, n, k, shares, correction):
    from ferrite_b200 import ops
    rng, on = np.random.default_rng(10), Device(torch, False)
    z = f32(np.argsort(rng.random((T, n)), 1) * (9.0 / n) - 4 + rng.normal(0, 0.2 / n, (T, n)))
    c = np.zeros(n)
    c[rng.integers(n)], c[rng.integers(n)] = 2.0, -2.0
    r = ops.route(on(z), n, k, on(c) if correction else None, "sigmoid", 0, 1.7, not shares, True)
    s = oracle.sigmoid(z)
    picks = np.argsort(-(s + c) if correction else -z, axis=-1, kind="stable")[:, :k]
    want = np.take_along_axis(s, picks, -1)
    want = (want / want.sum(-1, keepdims=True) if shares else want) * 1.7
    assert np.array_equal(to_numpy(r.ids), picks)
    np.testing.assert_allclose(to_numpy(r.weights), want, rtol=2e-5)
    assert np.array_equal(to_numpy(r.row_weights)[to_numpy(r.slots)], to_numpy(r.weights))


def test_sigmoids_that_round_to_one_are_told_apart(torch):
    from ferrite_b200 import ops
    z = np.array([[20.0, 31, 25, 40, 18]])
    r = ops.route(Device(torch, False)(z), 5, 3, None, "sigmoid", as_scored=True)
    assert to_numpy(r.ids).tolist() == [[3, 1, 2]] and np.abs(to_numpy(r.weights) - 1).max() < 1e-6


@pytest.mark.parametrize("T,n,k,K,m,bf16", [(1, 6, 2, 64, 32, True), (32, 10, 3, 320, 80, True), (300, 11, 4, 192, 48, True), (30, 5, 3, 60, 13, True), (100, 5, 3, 60, 13, False), (9, 1, 1, 64, 32, True), (80, 1, 1, 64, 32, True),
                                            (64, 7, 7, 256, 24, False), (700, 40, 8, 128, 512, True)])
def test_experts_weighted_on_their_inputs(torch, rt, T, n, k, K, m, bf16):
    from ferrite_b200.tensor import Tensor
    rng, kind = np.random.default_rng(11), "bf16" if bf16 else "fp32"
    w = {f"e{e}.{name}": rounded(rng.normal(0, 1.5 * shape[1] ** -0.5, shape), bf16) for e in range(n) for name, shape in (("up", (m, K)), ("down", (K, m)))}
    h, x = rounded(rng.normal(0, 1, (T, K)), bf16), f32(rng.normal(0, 1, (T, K)))
    z = f32(np.argsort(rng.random((T, n)), 1) * (5.0 / n) - 2.5)
    stack = lambda f: Tensor.of(rt, np.stack([f(e) for e in range(n)]), kind).T
    routes = Tensor.of(rt, z, "fp32").route(n, k, None, "sigmoid", as_scored=True, on_input=True)
    hd = Tensor.of(rt, h, kind)
    rows = hd.experts(routes, stack(lambda e: w[f"e{e}.up"]), stack(lambda e: w[f"e{e}.down"]), relu2=True)
    got, _ = Tensor.of(rt, x, "fp32").add_norm(Tensor.of(rt, np.ones((1, K)), "fp32"), 1e-3, dtype=kind, experts=(rows, routes))
    w["router"] = np.eye(n)
    picks, weights = oracle.route(z, w, "", dict(top=k))
    want = x.copy()
    for t in range(T):
        for e, s in zip(picks[t], weights[t]):
            want[t] += oracle.expert(s * h[t:t + 1], w, f"e{e}.")[0]
    assert np.abs(got.numpy()[0] - want).max() < (2e-2 if bf16 else 5e-6) * np.abs(want).max()


@pytest.mark.parametrize("T,n,k,K,m,limit", [(40, 5, 2, 64, 32, None), (200, 5, 2, 64, 32, 0.9), (50, 4, 2, 60, 13, 0.9)])
def test_gated_experts_take_weights_on_their_inputs_too(torch, rt, T, n, k, K, m, limit):
    from ferrite_b200.tensor import Tensor
    from oracle import vunadra
    rng = np.random.default_rng(12)
    w = {f"e{e}.{name}": rounded(rng.normal(0, 1.5 * shape[1] ** -0.5, shape), True) for e in range(n) for name, shape in (("gate", (m, K)), ("up", (m, K)), ("down", (K, m)))}
    h, z = rounded(rng.normal(0, 1, (T, K)), True), f32(np.argsort(rng.random((T, n)), 1) * (5.0 / n) - 2.5)
    stack = lambda f: Tensor.of(rt, np.stack([f(e) for e in range(n)])).T
    routes, hd = Tensor.of(rt, z, "fp32").route(n, k, None, "sigmoid", as_scored=True, on_input=True), Tensor.of(rt, h)
    rows = hd.experts(routes, stack(lambda e: np.concatenate([w[f"e{e}.gate"], w[f"e{e}.up"]])), stack(lambda e: w[f"e{e}.down"]), limit and (limit, vunadra.SLOPE)).numpy()[0]
    w["router"] = np.eye(n)
    picks, weights = oracle.route(z, w, "", dict(top=k))
    plain = lambda y, pre: oracle.linear(oracle.silu(oracle.linear(y, w, pre + "gate")) * oracle.linear(y, w, pre + "up"), w, pre + "down")
    slots = to_numpy(routes.slots)
    for t in range(T):
        for j in range(k):
            y, pre = weights[t, j] * h[t:t + 1], f"e{picks[t, j]}."
            want = (vunadra.expert(y, w, pre, limit) if limit else plain(y, pre))[0]
            assert np.abs(rows[slots[t, j]] - want).max() < 2e-2 * np.abs(want).max() + 1e-3


# ---- a layer's end

@pytest.mark.parametrize("cols,source,bf16", [(288, "bf16", True), (260, "fp32", True), (61, "fp32", False), (61, "bf16", True), (4096, "fp32", True), (5000, "fp32", False), (9000, "fp32", False)])
@pytest.mark.parametrize("T", [5, 600])
def test_gated_and_normed_branches(torch, cols, source, bf16, T):
    from ferrite_b200 import ops
    rng, on, src = np.random.default_rng(13), Device(torch, bf16), Device(torch, source == "bf16")
    T = T if cols < 1000 or T == 5 else 520
    x, g, b, post, w = (f32(rng.normal(0, 1, s)) for s in ((T, cols), (T, cols + 4), cols, cols, cols))
    y = rounded(rng.normal(0, 3, (T, cols)), source == "bf16")
    tol = 8e-3 if bf16 else 2e-5
    for gated, normed, last in ((1, 1, 1), (1, 0, 1), (0, 1, 1), (1, 1, 0)):
        out, h = on.f32(np.zeros((T, cols))), on(np.zeros((T, cols)))
        ops.add_norm(on.f32(x), out, src(y), None, w=on.f32(w) if last else None, eps=1e-2, h=h, gate=on.f32(g)[:, 4:] if gated else None, gate_bias=on.f32(b) if gated else None, post=on.f32(post) if normed else None)
        v = y * oracle.sigmoid(g[:, 4:] + b) if gated else y
        want = x + (oracle.rms(v, post, 1e-2) if normed else v)
        np.testing.assert_allclose(to_numpy(out), want, rtol=2e-5, atol=4e-5)
        np.testing.assert_allclose(to_numpy(h), oracle.rms(want, w, 1e-2) if last else want, rtol=tol, atol=tol)


def test_a_projection_of_any_width_leaves_aligned_rows(torch, rt):
    from ferrite_b200 import mixers
    from ferrite_b200.tensor import Tensor
    rng = np.random.default_rng(14)
    for K, N, kind in ((64, 102, "bf16"), (64, 96, "bf16"), (60, 13, "bf16"), (64, 103, "fp32")):
        h, w = rounded(rng.normal(0, 1, (9, K)), kind == "bf16"), rounded(rng.normal(0, 1, (N, K)), kind == "bf16")
        y = mixers.project(Tensor.of(rt, h, kind), Tensor.of(rt, w, kind).T)
        assert y.buf.stride(1) % 8 == 0 and y.buf.data_ptr() % 16 == 0 and y.shape == (1, 9, N)
        np.testing.assert_allclose(y.numpy()[0], h @ w.T, rtol=1e-4, atol=1e-4)
