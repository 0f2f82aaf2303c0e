"""The kernels of a grouped-query layer with experts, each alone, against plain numpy: attention within spans (both forms, every
size of the tensor-core kernel and the general one, keys planted at the edges), the projection's biases, norms, mixed values
and cache rows, the router's choices and places, the grouped matmuls, the layer's end, the embedding."""
import numpy as np
import pytest

from conftest import to_numpy
from oracle import labepel as oracle

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def torch(cuda):
    import torch
    return torch


def rounded(a, bf16):
    """a as the device holds it, in float64."""
    a = np.asarray(a, np.float32)
    if not bf16:
        return a.astype(np.float64)
    bits = np.ascontiguousarray(a).view(np.uint32)
    return ((bits + (0x7FFF + (bits >> 16 & 1))) >> 16 << 16).astype(np.uint32).view(np.float32).astype(np.float64)


class Device:
    def __init__(self, torch, bf16):
        self.torch, self.dtype = torch, torch.bfloat16 if bf16 else torch.float32

    def __call__(self, a, dtype=None):
        return self.torch.from_numpy(np.ascontiguousarray(np.asarray(a, np.float32))).to("cuda", dtype or self.dtype)

    def f32(self, a):
        return self(a, self.torch.float32)

    def i32(self, a):
        return self.torch.tensor(np.asarray(a), dtype=self.torch.int32, device="cuda")


# (heads, kv_heads, dim, vdim): every padded size of the tensor-core kernel, keys and values of no whole 16-column steps, more
# query heads a key head than a tile has rows; then what the general kernel takes (odd, or wider than 256)
SHAPES = [(12, 3, 112, 48), (4, 4, 64, 64), (6, 2, 40, 24), (32, 1, 128, 128), (4, 2, 136, 56), (2, 1, 256, 256), (40, 2, 72, 8), (3, 1, 64, 200), (5, 5, 128, 16)]
PLAIN = [(3, 1, 9, 7), (6, 3, 33, 65), (2, 2, 264, 72), (1, 1, 8, 300)]


def attention_case(torch, shape, bf16, T, places, span, rng, sink=True, gate=True, seqs=None, keys=None):
    """Device results and what they should be: one sequence's chunk at `places`, or a token of each of `seqs` sequences."""
    from ferrite_b200 import ops
    H, G, dim, vdim = shape
    on, n = Device(torch, bf16), max(places) + 1
    S, part = seqs or 1, n + 5
    q, cache = rounded(rng.normal(0, 1, (T, H, dim)), bf16), rounded(rng.normal(0, 1, (G, S * part, dim + vdim)), bf16)
    if keys is not None:
        keys(q, cache, part)
        q, cache = rounded(q, bf16), rounded(cache, bf16)
    zero = rng.normal(0.5, 1, H).astype(np.float32)
    g = rng.normal(0, 1.5, (T, H * vdim + T % 4)).astype(np.float32)  # (rows of gates that are aligned and rows that are not)
    scale = 1.3 / np.sqrt(dim)
    base = [u * part for u in range(T)] if seqs else None
    got = ops.heads_attention(on(q.reshape(T, H * dim)), on(cache), on.i32(base) if seqs else None, on.i32(places), H, vdim, scale, n, not seqs, span, on.f32(zero) if sink else None,
                              on.f32(g)[:, :H * vdim] if gate else None)
    want = np.zeros((T, H, vdim))
    for t, p in enumerate(places):
        lo, first = oracle.chunk_of(p, span) if span else 0, base[t] if seqs else 0
        for kv in range(G):
            mine = slice(kv * (H // G), (kv + 1) * (H // G))
            rows = cache[kv, first + lo:first + p + 1]
            s = q[t, mine] @ rows[:, :dim].T * scale
            m = np.maximum(s.max(-1), zero[mine] if sink else -np.inf)[:, None]
            e = np.exp(s - m)
            want[t, mine] = e @ rows[:, dim:] / (e.sum(-1, keepdims=True) + (np.exp(zero[mine, None] - m) if sink else 0))
    want = want.reshape(T, H * vdim)
    return to_numpy(got), want * oracle.sigmoid(np.float64(g[:, :H * vdim])) if gate else want


def close(got, want, bf16, what=None):
    assert np.abs(got - want).max() <= (1.5e-2 if bf16 else 2e-5) * max(np.abs(want).max(), 1e-3), what


@pytest.mark.parametrize("shape,bf16", [(s, True) for s in SHAPES + PLAIN] + [(s, False) for s in SHAPES[:3] + PLAIN])
def test_attention_of_a_prompt(torch, shape, bf16):
    rng = np.random.default_rng(0)
    for first, T, span in ((0, 150, 48), (0, 65, 64), (37, 70, 100), (200, 33, 0), (158, 2, 80), (79, 3, 80), (0, 40, 1)):
        got, want = attention_case(torch, shape, bf16, T, list(range(first, first + T)), span, rng)
        close(got, want, bf16, (first, T, span))
    got, want = attention_case(torch, shape, bf16, 20, list(range(600, 620)), 0, rng, sink=False, gate=False)  # (few tokens, many keys: a cluster shares them)
    close(got, want, bf16)


# prompts with tiles enough for the tcgen05 kernel: one group of pairs a CTA and two; pairs that fill a group's 128 rows and
# pairs that do not; keys and values of whole 64-column pieces, of 16-column steps and of neither; spans that begin inside tiles
@pytest.mark.parametrize("shape,cases", [((64, 32, 80, 48), ((0, 150, 48), (37, 200, 64), (190, 161, 0))), ((40, 40, 64, 64), ((0, 300, 100), (79, 257, 80))), ((90, 30, 40, 24), ((0, 130, 0), (60, 127, 33))),
                                         ((37, 37, 256, 128), ((0, 200, 77),)), ((48, 24, 136, 72), ((5, 260, 130),)), ((200, 2, 64, 32), ((0, 40, 0), (50, 40, 17))), ((74, 74, 8, 8), ((0, 70, 20), (3, 2, 1))),
                                         ((64, 32, 128, 128), ((0, 600, 0), (100, 640, 200))), ((32, 32, 192, 128), ((0, 640, 300),))])
def test_attention_of_a_long_prompt(torch, shape, cases):
    rng = np.random.default_rng(8)
    for first, T, span in cases:
        got, want = attention_case(torch, shape, True, T, list(range(first, first + T)), span, rng)
        close(got, want, True, (first, T, span))
    got, want = attention_case(torch, shape, True, T, list(range(first, first + T)), span, rng, sink=False, gate=False)
    close(got, want, True, (first, T, span))


def test_scores_that_grow_along_the_keys(torch):
    # each key outdoes the ones before, so the reference maximum moves at every tile, by different steps in different rows
    def plant(q, cache, part):
        cache[:, :, :64] = cache[:, :1, :64] * (1 + np.arange(part)[None, :, None] / 16)
        q[:] = cache[0, 0, :64] * np.linspace(0.2, 3, q.shape[0])[:, None, None]
    for T, shape in ((300, (32, 32, 64, 64)), (40, (4, 2, 64, 64))):
        got, want = attention_case(torch, shape, True, T, list(range(T)), 0, np.random.default_rng(9), keys=plant)
        close(got, want, True, T)


@pytest.mark.parametrize("shape,bf16", [(s, True) for s in SHAPES + PLAIN] + [(s, False) for s in SHAPES[:2] + PLAIN[:2]])
def test_attention_of_a_decode_step(torch, shape, bf16):
    rng = np.random.default_rng(1)
    for places, span in (([0, 1, 63, 64, 65, 127, 128, 300], 64), ([79, 80, 81, 5, 159, 160], 80), ([2000, 3], 0), ([700], 1000), ([1500, 40, 0], 512)):
        got, want = attention_case(torch, shape, bf16, len(places), places, span, rng, seqs=len(places))
        close(got, want, bf16, (places, span))


@pytest.mark.parametrize("prompt,shape", [(True, (4, 2, 64, 32)), (False, (4, 2, 64, 32)), (True, (74, 74, 64, 32))])
def test_a_key_at_the_edge_of_a_span(torch, prompt, shape):
    # the first key of a span, and the last of the one before, scored far above all others: the one decides, the other is unseen
    span = 40
    rng = np.random.default_rng(2)
    for first in (80, 160):
        for key, seen in ((first, True), (first - 1, False)):
            def plant(q, cache, part):
                q[:, :, :] = q[:1, :1, :]
                for u in range(1 if prompt else 8):
                    cache[:, u * part + key, :64] = q[0, 0] * 2
                    cache[:, u * part + key, 64:] = 8
            places = list(range(first, first + 8)) if prompt else [first + 3 * i for i in range(8)]
            got, want = attention_case(torch, shape, True, 8, places, span, rng, sink=False, gate=False, seqs=None if prompt else 8, keys=plant)
            close(got, want, True, (first, key))
            assert (np.abs(got - 8).max() < 0.1) == seen


@pytest.mark.parametrize("shape", [(12, 3, 112, 48), (3, 1, 9, 7), (2, 2, 300, 270)])
@pytest.mark.parametrize("source,bf16", [("fp32", True), ("fp32", False), ("bf16", True)])
def test_biases_norms_mixed_values_and_cache_rows(torch, shape, source, bf16):
    from ferrite_b200 import ops
    (H, G, dim, vdim), T, rows = shape, 37, 60
    rng, on = np.random.default_rng(3), Device(torch, bf16)
    n, wide = (H + G) * dim, G * vdim
    x, first = rounded(rng.normal(0, 1, (T, n + wide + 11)), source == "bf16"), rounded(rng.normal(0, 1, (T, wide + 5)), source == "bf16")
    b, fb, qn, kn = rng.normal(0, 1, n + wide), rng.normal(0, 1, wide), rng.normal(1, 0.3, dim), rng.normal(1, 0.3, dim)
    b, fb, qn, kn = (np.float64(np.float32(v)) for v in (b, fb, qn, kn))
    at = rng.permutation(rows)[:T].astype(np.int32)
    at[5], at[9] = -1, rows  # outside: not written
    src = Device(torch, source == "bf16")
    for norms, mixed in ((True, True), (False, False), (True, False)):
        cache, q = on(np.full((G, rows, dim + vdim), 7.0)), on(np.zeros((T, H * dim)))
        ops.heads_put(src(x), H, G, dim, vdim, on.i32(at), cache, q, on.f32(b), on.f32(qn) if norms else None, on.f32(kn) if norms else None, 1e-2,
                      src(first)[:, :wide] if mixed else None, on.f32(fb) if mixed else None, on.f32([0.3]) if mixed else None)
        heads = (x[:, :n] + b[:n]).reshape(T, H + G, dim)
        if norms:
            heads = np.concatenate([oracle.rms(heads[:, :H], qn, 1e-2), oracle.rms(heads[:, H:], kn, 1e-2)], 1)
        v = x[:, n:n + wide] + b[n:]
        if mixed:
            v = oracle.mix_values(v, first[:, :wide] + fb, np.float64(np.float32(0.3)))
        want = np.full((G, rows, dim + vdim), 7.0)
        for t in range(T):
            if 0 <= at[t] < rows:
                want[:, at[t], :dim], want[:, at[t], dim:] = heads[t, H:], v[t].reshape(G, vdim)
        tol = 5e-3 if bf16 else 2e-6
        np.testing.assert_allclose(to_numpy(q), heads[:, :H].reshape(T, H * dim), rtol=tol, atol=tol)
        np.testing.assert_allclose(to_numpy(cache), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("T,n,k", [(1, 6, 2), (7, 11, 4), (33, 128, 8), (64, 5, 5), (65, 130, 3), (200, 8, 2), (129, 1, 1), (700, 40, 32), (5, 50, 50), (130, 64, 64), (1500, 300, 6)])
def test_routes(torch, T, n, k):
    from ferrite_b200 import ops
    rng, on = np.random.default_rng(4), Device(torch, False)
    z, b = rng.integers(-6, 7, (T, n + 3)).astype(np.float64) / 2, rng.integers(-2, 3, n).astype(np.float64) / 2  # (many equal logits)
    r = ops.route(on(z)[:, :n], n, k, on(b))
    z = z[:, :n] + b
    picks = np.argsort(-z, axis=-1, kind="stable")[:, :k]
    e = np.exp(np.take_along_axis(z, picks, -1) - z.max(-1, keepdims=True))
    assert np.array_equal(to_numpy(r.ids), picks)
    np.testing.assert_allclose(to_numpy(r.weights), e / e.sum(-1, keepdims=True), rtol=1e-5, atol=1e-7)
    live, runs, slots = int(to_numpy(r.live)[0]), to_numpy(r.tile_expert), to_numpy(r.slots)
    experts = runs[:, 0]
    count = np.bincount(picks.reshape(-1), minlength=n)
    assert r.shared == (T <= 64) and live == ((count > 0) if r.shared else -(-count // r.tile)).sum() <= r.tiles
    assert (experts[live:] == n).all() and (np.diff(experts[:live]) >= 0).all()
    for i in range(live):
        mine = np.flatnonzero(experts[:live] == experts[i])
        assert runs[i, 1] == mine[0] and runs[i, 2] == len(mine)
    assert np.array_equal(experts[slots // r.tile], picks)
    if r.shared:
        assert np.array_equal(slots % r.tile, np.repeat(np.arange(T)[:, None], k, 1))
    else:
        assert len(set(slots.reshape(-1).tolist())) == T * k
        for dtype, cols in ((torch.bfloat16, 24), (torch.float32, 7), (torch.bfloat16, 9)):
            x = on(rng.integers(-99, 99, (T, cols + 8)), dtype)[:, :cols]
            out = ops.spread_rows(x, r, torch.zeros(r.tiles * r.tile, cols, dtype=dtype, device="cuda"))
            assert np.array_equal(to_numpy(out)[slots], np.repeat(to_numpy(x)[:, None], k, 1))


@pytest.mark.parametrize("T,n,k,K,m,N,bf16", [(1, 6, 2, 64, 32, 96, True), (32, 10, 3, 320, 80, 200, True), (17, 40, 8, 72, 48, 40, True), (64, 3, 1, 1024, 512, 512, True), (300, 11, 4, 192, 48, 264, True),
                                              (900, 2, 2, 128, 96, 128, True), (150, 70, 2, 136, 16, 72, True), (2000, 20, 3, 192, 160, 320, True), (30, 5, 3, 60, 13, 60, True), (100, 5, 3, 60, 13, 60, True),
                                              (9, 4, 2, 64, 32, 64, False), (120, 7, 2, 50, 21, 34, False)])
def test_experts(torch, T, n, k, K, m, N, bf16):
    from ferrite_b200.tensor import Runtime, Tensor
    rng, rt = np.random.default_rng(5), Runtime(0)
    on = Device(torch, bf16)
    w = {}
    for e in range(n):
        for name, shape in (("gate", (m, K)), ("up", (m, K)), ("down", (N, m))):
            w[f"e{e}.{name}"] = rounded(rng.normal(0, 1.5 * shape[1] ** -0.5, shape), bf16)
    h, z = rounded(rng.normal(0, 1, (T, K)), bf16), np.float64(np.float32(rng.normal(0, 1, (T, n))))
    tensor = lambda a, dtype="bf16" if bf16 else "fp32": Tensor(rt, a.shape[-2], a.shape[-1], batch=a.shape[0] if a.dim() == 3 else 1, dtype=dtype, buf=a.view(-1, *a.shape[-2:]))
    gate_up = tensor(on(np.stack([np.concatenate([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(n)]))).T
    down = tensor(on(np.stack([w[f"e{e}.down"] for e in range(n)]))).T
    routes = tensor(on.f32(z), "fp32").route(n, k)
    rows = tensor(on(h)).experts(routes, gate_up, down).numpy()[0]
    slots, picks = to_numpy(routes.slots), to_numpy(routes.ids)
    for t in range(T):
        for j in range(k):
            want = oracle.gated(h[t:t + 1], w, f"e{picks[t, j]}.")[0]
            assert np.abs(rows[slots[t, j]] - want).max() < (2e-2 if bf16 else 3e-6) * max(np.abs(want).max(), 0.5), (t, j)


@pytest.mark.parametrize("cols,source,bf16,T,k", [(288, "bf16", True, 9, 5), (260, "fp32", True, 9, 5), (61, "fp32", False, 9, 40), (61, "bf16", True, 9, 5), (128, "bf16", True, 3, 50), (4096, "bf16", True, 9, 5),
                                                  (2048, "bf16", True, 600, 2), (5120, "fp32", False, 9, 8), (9000, "bf16", True, 3, 2)])
def test_the_end_of_a_layer(torch, cols, source, bf16, T, k):
    from types import SimpleNamespace as NS
    from ferrite_b200 import ops
    rng, on, src = np.random.default_rng(6), Device(torch, bf16), Device(torch, source == "bf16")
    x, s1, s2, w = (np.float64(np.float32(rng.normal(0, 1, shape))) for shape in ((T, cols), cols, cols, cols))
    y, f = (rounded(rng.normal(0, 1, (T, cols)), source == "bf16") for _ in range(2))
    rows, slots, weights = rounded(rng.normal(0, 1, (T * k + 3, cols)), bf16), rng.permutation(T * k + 3)[:T * k].reshape(T, k), np.float64(np.float32(rng.uniform(0, 1, (T, k))))
    routes = NS(slots=on.i32(slots), weights=on.f32(weights), k=k)
    chosen = (rows[slots] * weights[..., None]).sum(1)
    for mixer, other, experts in ((1, 1, 1), (1, 0, 0), (0, 1, 0), (1, 0, 1), (0, 0, 0)):
        out, h = on.f32(np.zeros((T, cols))), on(np.zeros((T, cols)))
        ops.add_norm(on.f32(x), out, src(y) if mixer else None, on.f32(s1), src(f) if other else None, on.f32(s2), on(rows) if experts else None, routes if experts else None, on.f32(w), 1.0, 1e-3, h)
        want = x + mixer * y * s1 + (other * f + experts * chosen) * s2
        np.testing.assert_allclose(to_numpy(out), want, rtol=1e-5, atol=2e-5)
        tol = 6e-3 if bf16 else 1e-5
        np.testing.assert_allclose(to_numpy(h), oracle.rms(want, 1 + w, 1e-3), rtol=tol, atol=tol)


def test_embedding_and_places(torch):
    from ferrite_b200 import ops
    rng = np.random.default_rng(7)
    for bf16, cols in ((True, 96), (False, 61)):
        on = Device(torch, bf16)
        a, b = rounded(rng.normal(0, 1, (20, cols)), bf16), rounded(rng.normal(0, 1, (30, cols)), bf16)
        ids, places = [3, 0, 19, 25, 7], [0, 29, 4, 5, 1000]  # (outside: clamped)
        out = ops.embed(on(a), on.i32(ids), on(b), on.i32(places), on.f32(np.zeros((5, cols))))
        np.testing.assert_allclose(to_numpy(out), a[np.minimum(ids, 19)] + b[np.minimum(places, 29)], rtol=1e-6)
        out = ops.embed(on(a), on.i32(ids), None, None, on.f32(np.zeros((5, cols))))
        np.testing.assert_allclose(to_numpy(out), a[np.minimum(ids, 19)], rtol=1e-6)
