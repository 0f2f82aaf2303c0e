"""Ronavik: a decoder given by a list of layers over an fp32 residual stream, with an RMSNorm before and after every mixer and
feed-forward and each one's result gated by a sigmoid of what it read: x += norm_b(f(h) * sigmoid(W h + b)), h = norm(x).  Mixers:
`parallel`, attention weighted by sigmoids beside a gated linear recurrence, and `mamba2`, a state space; the feed-forward is a
mixture of experts with a squared ReLU, each weighted on its input by its router output's sigmoid, or left out.  There is no
rotation: a learned vector per place joins the embedding, which is the output layer too.

The module has a family's calls (models.py), with llama's names and meaning; what it shares with Llama - places, slots, prompts in
chunks, the greedy pick - is llama's own, the layer parts are mixers.py's.  Sizes and constants are config.json's.  Weights (names in
the checkpoint -> here): everything a mixer's layer projects its input to, side by side as `in` (the gate of the result first, then the
mixer's own: q, k, v, y, x; or in), likewise `mlp.in` (the gate, the router); a parallel mixer's two output matrices as one `mix.o`, the
recurrence's gates as the batch `mix.gates`; the experts as batches."""
from types import SimpleNamespace

import numpy as np
import torch

from . import llama, mixers, models
from .tensor import BFP, Tensor

REWINDS = False  # a recurrent state cannot be taken back to an earlier token: a slot's prefix is reused whole or not at all
MIXERS = {"parallel": (mixers.parallel, mixers.parallel_cache, mixers.parallel_width), "mamba2": (mixers.state_space, mixers.state_space_cache, mixers.state_space_width)}
DEFAULTS = dict(family="ronavik", places=4096, dtype="bf16", precision=None)


def model(**c):
    """A config from config.json's fields (vocab, width, norm, layers, max_positions) and this library's (places, dtype, precision)."""
    c = SimpleNamespace(**DEFAULTS | c)
    c.blocks = [models.sizes(e) for e in c.blocks]
    for i, b in enumerate(c.blocks):
        assert b.type in MIXERS, f"layer {i}: no mixer {b.type!r}: {', '.join(sorted(MIXERS))}"
        b.mlp, m = getattr(b, "mlp", None), b.mixer
        if b.type == "parallel":
            m.left.q_temp = getattr(m.left, "q_temp", None)
            assert m.left.heads % m.left.kv_heads == 0, f"layer {i}: whole groups of query heads per key head"
            assert m.right.width % m.right.blocks == 0 and m.right.conv >= 1, f"layer {i}: equal blocks of the recurrence's columns"
        else:
            assert m.heads % m.groups == 0 and m.heads * m.vdim % m.norm_groups == 0 and m.conv >= 1, f"layer {i}: whole groups of heads, equal parts of the norm"
        if b.mlp:
            assert b.mlp.kind == "moe", f"layer {i}: no feed-forward {b.mlp.kind!r}: moe"
            assert 1 <= b.mlp.router.top <= b.mlp.router.experts, f"layer {i}: {b.mlp.router.top} of {b.mlp.router.experts} experts"
    c.layers = len(c.blocks)
    return c


def config(j, places=4096):
    """A parsed config.json as a config."""
    return model(vocab=j["vocab"], dim=j["width"], eps=j["norm"]["eps"], blocks=j["layers"], positions=j["max_positions"], places=places)


def projections(c, l):
    """{op: (rows, columns)} of layer l's projections as x @ w takes them (experts: each)."""
    b, m, d = c.blocks[l], c.blocks[l].mixer, c.dim
    inner = m.left.heads * m.left.vdim + m.right.width if b.type == "parallel" else m.heads * m.vdim
    out = {"in": (d, d + MIXERS[b.type][2](m)), "mix.o": (inner, d)}
    return out | ({"mlp.in": (d, d + b.mlp.router.experts), "mlp.up": (d, b.mlp.expert.ff), "mlp.down": (b.mlp.expert.ff, d)} if b.mlp else {})


def precision(c, mode="bf16", kv=None):
    """{(op, block): (format, phases)} as llama.precision's: mode bf16, fp32 (everything in fp32), bfp8 or bfp4 (the block-float
    formats for the mixers' projections and the output layer; experts, routers and a recurrence's gates stay bf16, and so does a matrix
    without whole runs of 16 columns)."""
    assert kv in (None, "bf16", "fp32"), "keys and values are cached as the activations are kept"
    fmt = lambda k, n: "bf16" if mode in BFP and (n % 16 or k % 4) else mode
    p = {}
    for l in range(c.layers):
        p |= {(op, l): ("bf16" if mode in BFP and op.startswith("mlp.") else fmt(*shape), 4) for op, shape in projections(c, l).items()}
    p["head", None] = (fmt(c.dim, c.vocab), 4)
    p["act", None] = ("fp32" if mode == "fp32" else "bf16", None)
    return p


def weight_format(name, prec):
    """A weight's format on the device: the projections per prec, the vectors fp32, the rest as the activations are."""
    act = (prec or {}).get(("act", None), ("bf16",))[0]
    if name == "head":
        return (prec or {}).get(("head", None), (act,))[0]
    if name in ("embed", "pos"):
        return act
    layer, op = name.split(".", 1)
    if op in ("in", "mix.o", "mlp.in", "mlp.up", "mlp.down"):
        return (prec or {}).get((op, int(layer[1:])), (act,))[0]
    return act if op == "mix.gates" else "fp32"


def upload(rt, weights, prec=None):
    return finish(rt, llama.upload(rt, weights, prec, weight_format), prec)


def finish(rt, w, prec):
    """The output layer - the embedding, turned; a copy only in another format - and the layers' weights by layer."""
    f = weight_format("head", prec)
    w["head"] = w["embed"].T if f == w["embed"].dtype else w["embed"].T.cast(f).realize()
    llama.settle(rt, w)
    layers = 1 + max(int(n[1:].split(".")[0]) for n in w if n[0] == "l" and n[1:2].isdigit())
    w["_blocks"] = [llama.block(w, f"l{l}.") for l in range(layers)]
    return w


def with_precision(c, mode):
    """c as it computes under a mode of `precision` (what activations and caches are kept in), and that precision."""
    prec = precision(c, mode)
    return SimpleNamespace(**vars(c) | dict(dtype=prec["act", None][0], precision=prec)), prec


def weights(tensors, c):
    """{name: Weight} from a checkpoint's {name: (data, header entry)}."""
    from .checkpoint import join, leaf, rows, stack, turned
    w = {name: leaf(data, t, name.endswith(".conv")) for name, (data, t) in tensors.items()}
    for l, b in enumerate(c.blocks):
        pre = f"l{l}."
        mix = lambda *names: [w.pop(f"{pre}mix.{n}") for n in names]
        if b.type == "parallel":
            own = mix("left.q", "left.k", "left.v", "right.y", "right.x")
            w[pre + "mix.o"] = turned(join(*mix("left.o", "right.o")))
            w[pre + "mix.gates"], w[pre + "mix.gates.b"] = turned(rows(*mix("right.ra", "right.ri"))), join(*mix("right.ra.b", "right.ri.b"))
            for n in ("left.q.norm", "left.k.norm", "left.pb", "right.y.b", "right.x.b", "right.conv", "right.conv.b", "right.lam"):
                w[f"{pre}mix.{n.split('.', 1)[1]}"] = w.pop(f"{pre}mix.{n}")
        else:
            own = mix("in")
            w[pre + "mix.o"] = turned(w[pre + "mix.o"])
        w[pre + "in"] = turned(rows(w.pop(pre + "rg1"), *own))
        if b.mlp:
            expert = lambda n: [w.pop(f"{pre}mlp.e{e}.{n}") for e in range(b.mlp.router.experts)]
            w[pre + "mlp.up"], w[pre + "mlp.down"] = turned(stack(expert("up"))), turned(stack(expert("down")))
            w[pre + "mlp.in"] = turned(rows(w.pop(pre + "rg2"), w.pop(pre + "mlp.router")))
    return w


def layer(x, h, p, b, c, at, cache, norm):
    """One layer over the stream x and its normed rows h; the stream after it, and that normed for what comes next (norm: the next layer's
    weight, or the model's)."""
    ends = dict(eps=c.eps, dtype=c.dtype)
    joint = mixers.project(h, p["in"])
    y = MIXERS[b.type][0](joint[:, :, c.dim:], p, b.mixer, c.eps, at, cache)
    x, h = x.add_norm(p["norm2"] if b.mlp else norm, mixer=y, gate=joint[:, :, :c.dim], gate_bias=p["rg1.b"], post=p["norm1b"], **ends)
    if not b.mlp:
        return x, h
    joint = mixers.project(h, p["mlp.in"])
    _, experts = mixers.mixture(h, joint[:, :, c.dim:], p, "mlp.", b.mlp.router.top, scored="sigmoid", as_scored=True, on_input=True)
    return x.add_norm(norm, experts=experts, gate=joint[:, :, :c.dim], gate_bias=p["rg2.b"], post=p["norm2b"], **ends)


def forward(ids, places, w, c, caches, slots=None, every=False, length=None, residuals=None):
    """The logits for the token after ids, the tokens at places (llama.forward): every: all the tokens' (True), or those of
    the step's rows it names (int32, on the device).  residuals: a list that receives the stream after every layer."""
    rows, seen, _ = llama.around(w, c, places, caches.size, slots, length)
    at = SimpleNamespace(places=places, rows=rows, seen=seen, chunk=not slots and places.cols > 1, dead=caches.size // slots - 1 if slots else -1, dtype=c.dtype)
    norms = [p["norm1"] for p in w["_blocks"]] + [w["final.norm"]]
    x, h = w["embed"].embed(ids, w["pos"], places).add_norm(norms[0], c.eps, dtype=c.dtype)
    for b, p, cache, norm in zip(c.blocks, w["_blocks"], caches, norms[1:]):
        x, h = layer(x, h, p, b, c, at, cache, norm)
        if residuals is not None:
            residuals.append(x)
    if isinstance(every, Tensor):
        h = h.gather(every)
    elif not (slots or every):
        h = h[:, x.rows - 1:, :]
    return h.matmul(w["head"], dtype="fp32")


def kv_cache(c, size, zeros, slots=1):
    make = lambda shape, dtype=c.dtype: zeros(shape, dtype)
    return mixers.Caches(size, [MIXERS[b.type][1](b.mixer, size, make, slots) for b in c.blocks])


def slot(c, caches, u, slots):
    """Sequence u's part of caches made for several, in place."""
    return mixers.slot(caches, u, slots)


def random_weights(rt, c, prec=None, seed=0, scale=0.02):
    """Random weights in c's shapes made on the device: matrices N(0, scale), norms 1, small biases."""
    gen = torch.Generator(device=rt.device).manual_seed(seed)
    w = {}

    def matrix(name, n, k, batch=1):  # [k, n], each output column's weights together
        x = torch.empty(batch, n, k, dtype=torch.bfloat16, device=rt.device)
        for e in range(batch):
            x[e] = torch.empty(n, k, dtype=torch.float32, device=rt.device).normal_(0, scale, generator=gen)
        t = Tensor(rt, n, k, batch=batch, buf=x)
        f = weight_format(name, prec)
        w[name] = t.T if f == "bf16" else t.T.cast(f).realize()

    def vector(name, n, value, rows=1):
        w[name] = Tensor.of(rt, np.full((rows, n), value, np.float32), "fp32")

    for l, b in enumerate(c.blocks):
        pre, m = f"l{l}.", b.mixer
        for op, (k, n) in projections(c, l).items():
            matrix(pre + op, n, k, b.mlp.router.experts if op in ("mlp.up", "mlp.down") else 1)
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if b.mlp else ()):
            vector(pre + n, c.dim, 1.0)
        for n in ("rg1.b",) + (("rg2.b",) if b.mlp else ()):
            vector(pre + n, c.dim, 0.01)
        if b.type == "parallel":
            wide, part = m.right.width, m.right.width // m.right.blocks
            vector(pre + "mix.q.norm", m.left.dim, 1.0), vector(pre + "mix.k.norm", m.left.dim, 1.0), vector(pre + "mix.pb", m.left.heads, -4.0)
            matrix(pre + "mix.gates", 2 * part, part, m.right.blocks), vector(pre + "mix.gates.b", 2 * part, 0.01, m.right.blocks), vector(pre + "mix.lam", wide, 0.5)
            vector(pre + "mix.y.b", wide, 0.01), vector(pre + "mix.x.b", wide, 0.01), vector(pre + "mix.conv", wide, 0.3, m.right.conv), vector(pre + "mix.conv.b", wide, 0.01)
        else:
            inner, wide = m.heads * m.vdim, m.heads * m.vdim + 2 * m.groups * m.state
            vector(pre + "mix.conv", wide, 0.3, m.conv), vector(pre + "mix.conv.b", wide, 0.01), vector(pre + "mix.norm", inner, 1.0)
            vector(pre + "mix.dt_bias", m.heads, -2.0), vector(pre + "mix.A_log", m.heads, 0.5), vector(pre + "mix.D", m.heads, 1.0)
    vector("final.norm", c.dim, 1.0)
    for name, n in (("embed", c.vocab), ("pos", c.positions)):
        x = torch.empty(n, c.dim, dtype=torch.float32, device=rt.device).normal_(0, 1, generator=gen)
        w[name] = Tensor(rt, n, c.dim, dtype=c.dtype, buf=x.to(torch.float32 if c.dtype == "fp32" else torch.bfloat16).view(1, n, c.dim))
    return finish(rt, w, prec)
