"""Vunadra: a decoder given by a list of layers, some of which run several times in a row with the same weights (a loop).  A layer
is a token mixer and, unless left out, a feed-forward, each after an RMSNorm and added to an fp32 residual stream.  Mixers:
attention with a short convolution on queries, keys and values (`attention`), attention whose values are its keys, with joint norms,
capped scores and a window (`attention_2`), and attention over latents within a window (`latent_attention`); feed-forwards: a
GELU-gated one or a mixture of clamped experts, some of which give back their input.  The output layer is the embedding.

Each pass of the loop keeps caches of its own.  Before its first layer the stream becomes a matrix times itself beside the
embedding output, plus a vector of the pass.

The module has a family's calls (models.py), with llama's names and meaning; what it shares with Llama - places, slots,
prompts in chunks, the greedy pick - is llama's own, the layer parts are mixers.py's.  Sizes and constants are config.json's; the
experts' slope is the design's.  Weights (names in the checkpoint -> here): a mixer's projections side by side as `mix.in` (q, k, v;
q, k; q, dkv), their biases as `mix.b`, convolutions as `mix.conv`, gate | up as `mlp.gate_up` (experts: a batch), the router's
correction as `mlp.router.b`; the final norm's weight holds the logits' scale."""
from types import SimpleNamespace

import numpy as np
import torch

from . import llama, mixers, models
from .tensor import BFP, Tensor

REWINDS = False  # a convolution's state cannot be taken back to an earlier token: a slot's prefix is reused whole or not at all
GLU_SLOPE = 1.702
MIXERS = {"attention": (mixers.turned_attention, mixers.turned_cache), "attention_2": (mixers.turned_attention, mixers.turned_cache),
          "latent_attention": (mixers.latent_attention, mixers.latent_cache)}
DEFAULTS = dict(family="vunadra", places=4096, dtype="bf16", precision=None, loop=None, embed_scale=1.0, logit_scale=1.0)


def model(**c):
    """A config from config.json's fields (vocab, width, norm, layers, loop, scales) and this library's (places, dtype, precision)."""
    c = SimpleNamespace(**DEFAULTS | c)
    c.blocks = [models.sizes(e) for e in c.blocks]
    for i, b in enumerate(c.blocks):
        assert b.type in MIXERS, f"layer {i}: no mixer {b.type!r}: {', '.join(sorted(MIXERS))}"
        b.mlp, m = getattr(b, "mlp", None), b.mixer
        m.window = m.mask.size if getattr(m, "mask", None) else 0
        m.rot.scaling = getattr(m.rot, "scaling", None)
        if b.type == "latent_attention":
            assert m.rot.dims % 2 == 0 and m.rot.dims <= m.rot_dim, f"layer {i}: the turned columns are an even number of the key part's"
        else:
            m.keys_are_values = m.norm_all = b.type == "attention_2"
            m.conv, m.softcap = getattr(m, "conv", 0) or 0, getattr(m, "softcap", 0.0) or 0.0
            assert m.heads % m.kv_heads == 0, f"layer {i}: whole groups of query heads per key head"
            assert m.rot.dims % 2 == 0 and m.rot.dims <= m.dim, f"layer {i}: the turned columns are an even number of a head's"
            assert not m.keys_are_values or m.vdim == m.dim, f"layer {i}: values that are the keys are as wide"
        if b.mlp:
            assert b.mlp.kind in ("dense", "moe"), f"layer {i}: no feed-forward {b.mlp.kind!r}: dense, moe"
            if b.mlp.kind == "moe":
                r = b.mlp.router
                r.identity = getattr(r, "identity", 0) or 0
                assert 1 <= r.top <= r.experts + r.identity, f"layer {i}: {r.top} of {r.experts + r.identity} experts"
    c.layers = len(c.blocks)
    c.loop = models.sizes(c.loop) if isinstance(c.loop, dict) else c.loop
    assert not c.loop or 0 <= c.loop.start < c.loop.stop <= c.layers and c.loop.times >= 1, "a loop is a run of layers"
    c.runs = runs(c)
    return c


def runs(c):
    """The layer runs in order: (layer, the number of the pass that begins with it or None)."""
    if not c.loop:
        return [(l, None) for l in range(c.layers)]
    a, b = c.loop.start, c.loop.stop
    return [(l, None) for l in range(a)] + [(l, t if l == a else None) for t in range(c.loop.times) for l in range(a, b)] + [(l, None) for l in range(b, c.layers)]


def config(j, places=4096):
    """A parsed config.json as a config."""
    return model(vocab=j["vocab"], dim=j["width"], eps=j["norm"]["eps"], blocks=j["layers"], loop=j.get("loop"), embed_scale=j["embedding"]["scale"], logit_scale=j["logit_scale"], places=places)


def projections(c, l):
    """{op: (rows, columns)} of layer l's projections as x @ w takes them."""
    b, m, d = c.blocks[l], c.blocks[l].mixer, c.dim
    wide = m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim if b.type == "latent_attention" else mixers.turned_width(m)
    ff = b.mlp and (b.mlp.ff if b.mlp.kind == "dense" else b.mlp.expert.ff)
    return {"mix.in": (d, wide), "mix.o": (m.heads * m.vdim, d)} | ({"mlp.gate_up": (d, 2 * ff), "mlp.down": (ff, d)} if b.mlp else {})


def precision(c, mode="bf16", kv=None):
    """{(op, block): (format, phases)} as llama.precision's: mode bf16, fp32 (everything in fp32), bfp8 or bfp4 (the block-float
    formats for the projections and dense feed-forwards; experts, routers and a head's own matrices stay bf16, and so does a matrix
    without whole runs of 16 columns)."""
    assert kv in (None, "bf16", "fp32"), "keys, values and latents are cached as the activations are kept"
    fmt = lambda k, n: "bf16" if mode in BFP and (n % 16 or k % 4) else mode
    p = {}
    for l, b in enumerate(c.blocks):
        for op, shape in projections(c, l).items():
            experts = op.startswith("mlp.") and b.mlp.kind == "moe" and mode in BFP
            p[op, l] = ("bf16" if experts else fmt(*shape), 4)
    p["loop.in", None], p["head", None] = (fmt(2 * c.dim, c.dim), 4), (fmt(c.dim, c.vocab), 4)
    p["act", None] = ("fp32" if mode == "fp32" else "bf16", None)
    return p


def weight_format(name, prec):
    """A weight's format on the device: the projections per prec, the vectors fp32, the rest as the activations are."""
    act = (prec or {}).get(("act", None), ("bf16",))[0]
    if name in ("head", "loop.in"):
        return (prec or {}).get((name, None), (act,))[0]
    if name == "embed" or name.endswith((".router", ".uk", ".uv")):
        return act
    if name.endswith((".in", ".o", ".gate_up", ".down")):
        layer, op = name.split(".", 1)
        return (prec or {}).get((op, int(layer[1:])), (act,))[0]
    return "fp32"


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
    from .checkpoint import batched, columns_together, join, leaf, rows, scaled, stack, turned
    w = {name: leaf(data, t, name.endswith(".conv")) for name, (data, t) in tensors.items()}
    for l, b in enumerate(c.blocks):
        pre, m = f"l{l}.", b.mixer
        mix = lambda names, end="": [w.pop(f"{pre}mix.{n}{end}") for n in names]
        if b.type == "latent_attention":
            w[pre + "mix.in"] = turned(rows(*mix(("q", "dkv"))))
            w[pre + "mix.uk"] = columns_together(batched(w[pre + "mix.uk"], m.heads))
            w[pre + "mix.uv"] = turned(batched(w[pre + "mix.uv"], m.heads))
        else:
            names = "qk" if m.keys_are_values else "qkv"
            w[pre + "mix.in"] = turned(rows(*mix(names)))
            if pre + "mix.q.b" in w:
                w[pre + "mix.b"] = join(*mix(names, ".b"))
            if m.conv:
                w[pre + "mix.conv"] = join(*mix(names, ".conv"))
        w[pre + "mix.o"] = turned(w[pre + "mix.o"])
        if b.mlp and b.mlp.kind == "dense":
            w[pre + "mlp.gate_up"] = turned(rows(w.pop(pre + "mlp.gate"), w.pop(pre + "mlp.up")))
            w[pre + "mlp.gate_up.b"] = join(w.pop(pre + "mlp.gate.b"), w.pop(pre + "mlp.up.b"))
            w[pre + "mlp.down"] = turned(w[pre + "mlp.down"])
        elif b.mlp:
            expert = lambda n: [w.pop(f"{pre}mlp.e{e}.{n}") for e in range(b.mlp.router.experts)]
            w[pre + "mlp.gate_up"] = turned(stack([rows(g, u) for g, u in zip(expert("gate"), expert("up"))]))
            w[pre + "mlp.down"] = turned(stack(expert("down")))
            w[pre + "mlp.router"], w[pre + "mlp.router.b"] = turned(w[pre + "mlp.router"]), w.pop(pre + "mlp.correction")
    if c.loop:
        w["loop.in"] = turned(w["loop.in"])
    w["final.norm"] = scaled(w["final.norm"], c.logit_scale)
    return w


def layer(x, h, p, b, c, at, cache, norm, into=None):
    """One layer over the stream x and its normed rows h; the stream after it, and what comes next reads: that normed by norm, or
    (None) as it is, into `into` where given."""
    y = MIXERS[b.type][0](h, p, b.mixer, c.eps, at, cache)
    ends = dict(eps=c.eps, dtype=c.dtype)
    if not b.mlp:
        return x.add_norm(norm, mixer=y, mixer_bias=p.get("mix.o.b"), into=into, **ends)
    x, h = x.add_norm(p["norm2"], mixer=y, mixer_bias=p.get("mix.o.b"), **ends)
    if b.mlp.kind == "dense":
        return x.add_norm(norm, mixer=mixers.gelu_mlp(h, p, "mlp."), mixer_bias=p["mlp.down.b"], into=into, **ends)
    r = b.mlp.router
    logits = h.matmul(p["mlp.router"], dtype="fp32")
    _, experts = mixers.mixture(h, logits, p, "mlp.", r.top, scored="softmax", identity=r.identity, scale=r.scale, clamp=(b.mlp.expert.limit, GLU_SLOPE))
    return x.add_norm(norm, experts=experts, own=h, into=into, **ends)


def forward(ids, places, w, c, caches, slots=None, every=False, length=None, residuals=None):
    """The logits for the token after ids, the tokens at places (llama.forward): every: all the tokens' (True), or those of
    the step's rows it names (int32, on the device).  residuals: a list that receives the stream after every layer run."""
    rows, seen, _ = llama.around(w, c, places, caches.size, slots, length)
    at = SimpleNamespace(places=places, rows=rows, seen=seen, chunk=not slots and places.cols > 1, dead=caches.size // slots - 1 if slots else -1)
    x = w["embed"].embed(ids, scale=c.embed_scale)
    beside = None
    if c.loop:  # the stream as a pass finds it | the embedding output
        beside = Tensor(x.rt, x.rows, 2 * c.dim, dtype=c.dtype)
        x.add_norm(None, 0.0, dtype=c.dtype, into=beside[:, :, c.dim:])

    def reads(i):  # the norm before layer run i (or the end), and, where it begins a pass, where it finds the stream
        if i == len(c.runs):
            return w["final.norm"], None
        l, t = c.runs[i]
        return (w["_blocks"][l]["norm1"], None) if t is None else (None, beside[:, :, :c.dim])

    norm, into = reads(0)
    x, h = x.add_norm(norm, c.eps, dtype=c.dtype, into=into)
    for i, ((l, t), cache) in enumerate(zip(c.runs, caches)):
        p = w["_blocks"][l]
        if t is not None:
            x, h = beside.matmul(w["loop.in"], dtype="fp32").add_norm(p["norm1"], c.eps, dtype=c.dtype, mixer_bias=w["loop.step"][t:t + 1, :])
        norm, into = reads(i + 1)
        x, h = layer(x, h, p, c.blocks[l], c, at, cache, norm, into)
        if residuals is not None:
            residuals.append(x)
    if isinstance(every, Tensor):
        h = h.gather(every)
    elif not (slots or every):
        h = h[:, x.rows - 1:, :]
    return h.matmul(w["head"], dtype="fp32")


def kv_cache(c, size, zeros, slots=1):
    """What each layer run keeps: a pass of the loop has its own."""
    make = lambda shape, dtype=c.dtype: zeros(shape, dtype)
    return mixers.Caches(size, [MIXERS[c.blocks[l].type][1](c.blocks[l].mixer, size, make, slots) for l, _ in c.runs])


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
        pre, m, r = f"l{l}.", b.mixer, b.mlp.router if b.mlp and b.mlp.kind == "moe" else None
        for op, (k, n) in projections(c, l).items():
            matrix(pre + op, n, k, r.experts if r and op.startswith("mlp.") else 1)
        vector(pre + "norm1", c.dim, 1.0)
        if b.type == "latent_attention":
            vector(pre + "mix.dkv.norm", m.kv_rank, 1.0)
            matrix(pre + "mix.uk", m.kv_rank, m.dim, m.heads), matrix(pre + "mix.uv", m.vdim, m.kv_rank, m.heads)
        elif b.type == "attention":
            vector(pre + "mix.conv", mixers.turned_width(m), 0.4, max(m.conv, 1))
        else:
            vector(pre + "mix.b", mixers.turned_width(m), 0.01), vector(pre + "mix.o.b", c.dim, 0.01)
            vector(pre + "mix.q.norm", m.heads * m.dim, 1.0), vector(pre + "mix.k.norm", m.kv_heads * m.dim, 1.0)
        if b.mlp:
            vector(pre + "norm2", c.dim, 1.0)
        if r:
            matrix(pre + "mlp.router", r.experts + r.identity, c.dim), vector(pre + "mlp.router.b", r.experts + r.identity, 0.0)
        elif b.mlp:
            vector(pre + "mlp.gate_up.b", 2 * b.mlp.ff, 0.01), vector(pre + "mlp.down.b", c.dim, 0.01)
    if c.loop:
        matrix("loop.in", c.dim, 2 * c.dim), vector("loop.step", c.dim, 0.1, c.loop.times)
    vector("final.norm", c.dim, c.logit_scale)
    embed = torch.empty(c.vocab, c.dim, dtype=torch.float32, device=rt.device).normal_(0, 1, generator=gen)
    w["embed"] = Tensor(rt, c.vocab, c.dim, dtype=c.dtype, buf=embed.to(torch.float32 if c.dtype == "fp32" else torch.bfloat16).view(1, c.vocab, c.dim))
    return finish(rt, w, prec)
