"""Labepel: a decoder given by a list of layers whose mixer and feed-forward read the same normed rows and are added to an fp32
residual stream together, each scaled by column.  The mixer is grouped-query attention within spans of the sequence (no
rotation: a learned vector per place joins the embedding), with biases, query and key norms, values mixed with the first
layer's, a sink in the softmax and an output gate; the feed-forward is a mixture of experts with a shared one, or left out.
The output layer is the embedding.

The module has a family's calls (models.py), with llama's names and meaning; what it shares with Llama - places, slots,
prompts in chunks, the greedy pick - is llama's own, the layer parts are mixers.py's.  Sizes and constants are config.json's.
Weights (names in the checkpoint -> here): everything a layer projects its input to, side by side as `in` (q, k, v, g and the
router; in block floats the router stays on its own), the three biases as `mix.b`, the experts' gate | up and down as the
batches `mlp.gate_up` and `mlp.down`, the shared expert's as `mlp.shared.gate_up`."""
from types import SimpleNamespace

import numpy as np
import torch

from . import llama, mixers, models
from .tensor import BFP, Tensor

DEFAULTS = dict(family="labepel", places=4096, dtype="bf16", precision=None)
SINK = 0.0  # every head's: one more term exp(0) in the softmax's denominator


def model(**c):
    """A config from config.json's fields (vocab, width, norm, layers, max_positions) and this library's (places, dtype, precision)."""
    c = SimpleNamespace(**DEFAULTS | c)
    c.blocks = [models.sizes(e) for e in c.blocks]
    mixing = None  # the first layer whose values later ones mix with theirs
    for i, b in enumerate(c.blocks):
        assert b.type == "attention", f"layer {i}: no mixer {b.type!r}: attention"
        b.mlp, m = getattr(b, "mlp", None), b.mixer
        m.v_mix = getattr(m, "v_mix", False)
        assert m.heads % m.kv_heads == 0 and m.mask.size >= 1, f"layer {i}: whole groups of query heads per key head, spans of at least a place"
        if m.v_mix:
            mixing = mixing or m
            assert m.kv_heads * m.vdim == mixing.kv_heads * mixing.vdim, f"layer {i}: mixed values are as wide as the first layer's"
        if b.mlp:
            assert b.mlp.kind == "moe", f"layer {i}: no feed-forward {b.mlp.kind!r}: moe"
            b.mlp.shared = getattr(b.mlp, "shared", None)
            assert 1 <= b.mlp.router.top <= b.mlp.router.experts, f"layer {i}: {b.mlp.router.top} of {b.mlp.router.experts} experts"
    c.layers = len(c.blocks)
    return c


def config(j, places=4096):
    """A parsed config.json as a config."""
    return model(vocab=j["vocab"], dim=j["width"], eps=j["norm"]["eps"], blocks=j["layers"], positions=j["max_positions"], places=places)


def projections(c, l):
    """{op: (rows, columns)} of layer l's projections as x @ w takes them."""
    b, m, d = c.blocks[l], c.blocks[l].mixer, c.dim
    out = {"in": (d, mixers.heads_width(m)), "mix.o": (m.heads * m.vdim, d)}
    if b.mlp:
        out |= {"mlp.gate_up": (d, 2 * b.mlp.expert.ff), "mlp.down": (b.mlp.expert.ff, d)}
        if b.mlp.shared:
            out |= {"mlp.shared.gate_up": (d, 2 * b.mlp.shared.ff), "mlp.shared.down": (b.mlp.shared.ff, d)}
    return out


def precision(c, mode="bf16", kv=None):
    """{(op, block): (format, phases)} as llama.precision's: mode bf16, fp32 (everything in fp32), bfp8 or bfp4 (the block-float
    formats for the projections and experts; the router stays bf16, and so does a matrix without whole runs of 16 columns)."""
    assert kv in (None, "bf16", "fp32"), "keys and values are cached as the activations are kept"
    fmt = lambda k, n: "bf16" if mode in BFP and (n % 16 or k % 4) else mode
    p = {}
    for l in range(c.layers):
        shapes = projections(c, l)
        p |= {(op, l): (fmt(*shape), 4) for op, shape in shapes.items()}
        both = {"mlp.gate_up", "mlp.down"} & set(shapes)
        if any(p[op, l][0] != mode for op in both):  # (an expert's two matrices go through the same kernels)
            p |= {(op, l): ("bf16", 4) for op in both}
    p["head", None] = (fmt(c.dim, c.vocab), 4)
    p["act", None] = ("fp32" if mode == "fp32" else "bf16", None)
    return p


def weight_format(name, prec):
    """A weight's format on the device: the projections per prec, the vectors fp32, the rest as the activations are."""
    act = (prec or {}).get(("act", None), ("bf16",))[0]
    if name == "head":
        return (prec or {}).get(("head", None), (act,))[0]
    if name in ("embed", "pos") or name.endswith(".router"):
        return act
    if name.startswith("l") and name.endswith((".in", ".o", ".gate_up", ".down")):
        layer, op = name.split(".", 1)
        return (prec or {}).get((op, int(layer[1:])), (act,))[0]
    return "fp32"


def routed_apart(l, prec):
    """Whether layer l's router is a matrix of its own: beside a joint projection in block floats it would be rounded too."""
    return weight_format(f"l{l}.in", prec) in BFP


def upload(rt, weights, prec=None):
    from .checkpoint import rows, turned
    w = dict(weights)
    for name in [n for n in w if n.endswith(".in")]:
        router = name.removesuffix("in") + "mlp.router"
        if router in w and not routed_apart(int(name[1:].split(".")[0]), prec):
            w[name] = rows(w[name], w.pop(router))
        elif router in w:
            w[router] = turned(w[router])
        w[name] = turned(w[name])
    w = llama.upload(rt, w, prec, weight_format)
    return finish(rt, w, prec)


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
    w = {name: leaf(data, t) for name, (data, t) in tensors.items()}
    for l, b in enumerate(c.blocks):
        pre = f"l{l}."
        w[pre + "in"] = rows(*(w.pop(f"{pre}mix.{n}") for n in "qkvg"))
        w[pre + "mix.b"] = join(*(w.pop(f"{pre}mix.{n}.b") for n in "qkv"))
        w[pre + "mix.o"] = turned(w[pre + "mix.o"])
        if b.mlp:
            expert = lambda n: [w.pop(f"{pre}mlp.e{e}.{n}") for e in range(b.mlp.router.experts)]
            w[pre + "mlp.gate_up"] = turned(stack([rows(g, u) for g, u in zip(expert("gate"), expert("up"))]))
            w[pre + "mlp.down"] = turned(stack(expert("down")))
            if b.mlp.shared:
                w[pre + "mlp.shared.gate_up"] = turned(rows(w.pop(pre + "mlp.shared.gate"), w.pop(pre + "mlp.shared.up")))
                w[pre + "mlp.shared.down"] = turned(w[pre + "mlp.shared.down"])
    return w


def layer(x, h, p, b, c, at, cache, norm):
    """One layer over its normed input h: mixer and feed-forward side by side; the stream after it, and that normed for what
    comes next (norm: the next layer's weight, or the model's)."""
    joint = h.matmul(p["in"], dtype="fp32").realize()
    y = mixers.heads_attention(joint, p, b.mixer, c.eps, at, cache, SINK)
    shared = experts = None
    if b.mlp:
        n = b.mlp.router.experts
        logits = h.matmul(p["mlp.router"], dtype="fp32") if "mlp.router" in p else joint[:, joint.cols - n:]
        shared, experts = mixers.mixture(h, logits, p, "mlp.", b.mlp.router.top)
    return x.add_norm(norm, c.eps, plus=1.0, dtype=c.dtype, mixer=y, mixer_scale=p["ls1"], other=shared, other_scale=p.get("ls2"), experts=experts)


def forward(ids, places, w, c, caches, slots=None, every=False, length=None, residuals=None):
    """The logits for the token after ids, the tokens at places (llama.forward): every: all the tokens' (True), or those of
    the step's rows it names (int32, on the device).  residuals: a list that receives the stream after every layer."""
    rows, seen, _ = llama.around(w, c, places, caches.size, slots, length)
    at = SimpleNamespace(places=places, rows=rows, seen=seen, chunk=not slots and places.cols > 1, first=None)
    norms = [p["norm1"] for p in w["_blocks"]] + [w["final.norm"]]
    x, h = w["embed"].embed(ids, w["pos"], places).add_norm(norms[0], c.eps, plus=1.0, dtype=c.dtype)
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
    return mixers.Caches(size, [mixers.heads_cache(b.mixer, size, make, slots) for b in c.blocks])


def slot(c, caches, u, slots):
    """Sequence u's part of caches made for several, in place."""
    return mixers.slot(caches, u, slots)


def random_weights(rt, c, prec=None, seed=0, scale=0.02):
    """Random weights in c's shapes made on the device: matrices N(0, scale), norms 1 (stored around zero), small biases."""
    gen = torch.Generator(device=rt.device).manual_seed(seed)
    w = {}

    def matrix(name, n, k, batch=1):  # [k, n], each output column's weights together
        x = torch.empty(batch, n, k, dtype=torch.bfloat16, device=rt.device)
        for e in range(batch):
            x[e] = torch.empty(n, k, dtype=torch.float32, device=rt.device).normal_(0, scale, generator=gen)
        t = Tensor(rt, n, k, batch=batch, buf=x)
        f = weight_format(name, prec)
        w[name] = t.T if f == "bf16" else t.T.cast(f).realize()

    def vector(name, n, value):
        w[name] = Tensor.of(rt, np.full((1, n), value, np.float32), "fp32")

    for l, b in enumerate(c.blocks):
        pre, m, shapes = f"l{l}.", b.mixer, projections(c, l)
        vector(pre + "norm1", c.dim, 0.0), vector(pre + "ls1", c.dim, 0.5), vector(pre + "mix.b", (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim, 0.01)
        vector(pre + "mix.q.norm", m.dim, 1.0), vector(pre + "mix.k.norm", m.dim, 1.0), vector(pre + "mix.vmix", 1, 0.3)
        router = b.mlp.router.experts if b.mlp else 0
        for op, (k, n) in shapes.items():
            experts = b.mlp.router.experts if op in ("mlp.gate_up", "mlp.down") else 1
            matrix(pre + op, n + (router if op == "in" and not routed_apart(l, prec) else 0), k, experts)
        if b.mlp:
            vector(pre + "ls2", c.dim, 0.5), vector(pre + "mlp.router.b", router, 0.0)
            if routed_apart(l, prec):
                matrix(pre + "mlp.router", router, c.dim)
    vector("final.norm", c.dim, 0.0)
    for name, n in (("embed", c.vocab), ("pos", c.positions)):
        x = torch.empty(n, c.dim, dtype=torch.float32, device=rt.device).normal_(0, 1, generator=gen)
        w[name] = Tensor(rt, n, c.dim, dtype=c.dtype, buf=x.to(torch.float32 if c.dtype == "fp32" else torch.bfloat16).view(1, n, c.dim))
    return finish(rt, w, prec)
