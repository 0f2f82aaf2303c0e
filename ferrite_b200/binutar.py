"""Binutar: a decoder given by a list of layers, each with a token mixer - attention over latents (with a query latent, a
sink and an output gate per head) or linear attention with a fixed decay per head - and, unless left out, a clamped gated
MLP.  A Dynamic Tanh stands before and after each of the two, the residual stream is fp32, and the model ends in one more
Dynamic Tanh and an output layer of its own.

The module has a family's calls (models.py), with llama's names and meaning; what it shares with Llama - places, slots,
prompts in chunks, the greedy pick - is llama's own.  Sizes and constants are config.json's; the gated unit's slope is the
design's.  Weights (names in the checkpoint -> here): a latent mixer's dq, dkv and g side by side as `mix.in`, a linear
mixer's q, k, v and g as `mix.qkvg`, gate and up as `gate_up`."""
from types import SimpleNamespace

import numpy as np
import torch

from . import llama, mixers, models
from .tensor import BFP, Tensor

REWINDS = False  # a linear mixer's state cannot be taken back to an earlier token: a slot's prefix is reused whole or not at all
GLU_SLOPE = 1.702
MIXERS = {"latent_attention": (mixers.latent_attention, mixers.latent_cache), "lightning": (mixers.decay_attention, mixers.decay_cache)}
DEFAULTS = dict(family="binutar", places=4096, dtype="bf16", precision=None)


def model(**c):
    """A config from config.json's fields (vocab, width, norm, layers) and this library's (places, dtype, precision)."""
    c = SimpleNamespace(**DEFAULTS | c)
    c.blocks = [models.sizes(e) for e in c.blocks]
    for i, b in enumerate(c.blocks):
        assert b.type in MIXERS, f"layer {i}: no mixer {b.type!r}: {', '.join(sorted(MIXERS))}"
        b.mlp = getattr(b, "mlp", None)
        assert b.mlp is None or b.mlp.kind == "dense", f"layer {i}: no feed-forward {b.mlp.kind!r}: dense"
        if b.type == "latent_attention":
            m = b.mixer
            m.rot.scaling = getattr(m.rot, "scaling", None)
            assert m.rot.dims % 2 == 0 and m.rot.dims <= m.rot_dim, f"layer {i}: the turned columns are an even number of the key part's"
        else:
            assert len(b.mixer.decay) == b.mixer.heads, f"layer {i}: a decay a head"
    c.layers = len(c.blocks)
    return c


def config(j, places=4096):
    """A parsed config.json as a config."""
    return model(vocab=j["vocab"], dim=j["width"], eps=j["norm"]["eps"], blocks=j["layers"], places=places)


def projections(c, l):
    """{op: (rows, columns)} of layer l's projections as x @ w takes them."""
    b, m, d = c.blocks[l], c.blocks[l].mixer, c.dim
    if b.type == "latent_attention":
        out = {"in": (d, m.q_rank + m.kv_rank + m.rot_dim + m.heads), "uq": (m.q_rank, m.heads * (m.dim + m.rot_dim))}
    else:
        out = {"qkvg": (d, 2 * m.heads * (m.dim + m.vdim))}
    return out | {"o": (m.heads * m.vdim, d)} | ({"gate_up": (d, 2 * b.mlp.ff), "down": (b.mlp.ff, d)} if b.mlp else {})


def precision(c, mode="bf16", kv=None):
    """{(op, block): (format, phases)} as llama.precision's: mode bf16, fp32 (everything in fp32), bfp8 or bfp4 (the block-float
    formats for the large projections; a head's own matrices, which act on the query and the weighted latents, stay bf16, and
    so does a matrix that has no whole runs of 16 columns)."""
    assert kv in (None, "bf16", "fp32"), "the latents are cached as the activations are kept"
    fmt = lambda k, n: "bf16" if mode in BFP and (n % 16 or k % 4) else mode
    p = {(op, l): (fmt(*shape), 4) for l in range(c.layers) for op, shape in projections(c, l).items()}
    p["head", None] = (fmt(c.dim, c.vocab), 4)
    p["act", None] = ("fp32" if mode == "fp32" else "bf16", None)
    return p


def weight_format(name, prec):
    """A weight's format on the device: the projections per prec, the vectors fp32, the rest as the activations are."""
    act = (prec or {}).get(("act", None), ("bf16",))[0]
    if name == "head":
        return (prec or {}).get(("head", None), (act,))[0]
    op = name.split(".")[-1]
    if name.startswith("l") and op in ("in", "uq", "o", "qkvg", "gate_up", "down"):
        return (prec or {}).get((op, int(name.split(".")[0][1:])), (act,))[0]
    return "fp32" if op in ("norm", "norm1", "norm2", "norm1b", "norm2b", "b", "alpha", "sink") else act


def upload(rt, weights, prec=None):
    return llama.upload(rt, weights, prec, weight_format)


def with_precision(c, mode):
    """c as it computes under a mode of `precision` (what activations and caches are kept in), and that precision."""
    prec = precision(c, mode)
    c = SimpleNamespace(**vars(c) | dict(dtype=prec["act", None][0], precision=prec))
    return c, prec


def fuse(w, c):
    """The checkpoint's matrices as the mixers take them: x @ w with w turned (a view: each output column's weights stay
    together, as the file has them), joint projections side by side, a head's own matrices as a batch."""
    from .checkpoint import batched, columns_together, rows, turned
    for l, b in enumerate(c.blocks):
        pre, m = f"l{l}.", b.mixer
        if b.type == "latent_attention":
            w[pre + "mix.in"] = turned(rows(w.pop(pre + "mix.dq"), w.pop(pre + "mix.dkv"), w.pop(pre + "mix.g")))
            w[pre + "mix.uq"] = turned(w[pre + "mix.uq"])
            w[pre + "mix.uk"] = columns_together(batched(w[pre + "mix.uk"], m.heads))
            w[pre + "mix.uv"] = turned(batched(w[pre + "mix.uv"], m.heads))
        else:
            w[pre + "mix.qkvg"] = turned(rows(*(w.pop(pre + "mix." + n) for n in "qkvg")))
        w[pre + "mix.o"] = turned(w[pre + "mix.o"])
        if b.mlp:
            w[pre + "mlp.gate_up"] = turned(rows(w.pop(pre + "mlp.gate"), w.pop(pre + "mlp.up")))
            w[pre + "mlp.down"] = turned(w[pre + "mlp.down"])
    w["head"] = turned(w["head"])
    return w


def weights(tensors, c):
    """{name: Weight} from a checkpoint's {name: (data, header entry)}."""
    from .checkpoint import leaf
    return fuse({name: leaf(data, t) for name, (data, t) in tensors.items()}, c)


def layer(x, p, b, c, at, cache):
    """One layer: the mixer, then the MLP if the layer has one, each between two Dynamic Tanhs and added to the residual."""
    run = MIXERS[b.type][0]
    x = x + mixers.dyt(run(mixers.dyt(x, p, "norm1").cast(c.dtype), p, b.mixer, c.eps, at, cache), p, "norm1b")
    if not b.mlp:
        return x
    h = mixers.dyt(x, p, "norm2").cast(c.dtype)
    return x + mixers.dyt(mixers.clamped_mlp(h, p, "mlp.", b.mlp.limit, GLU_SLOPE), p, "norm2b")


def forward(ids, places, w, c, caches, slots=None, every=False, length=None):
    """The logits for the token after ids, the tokens at places (llama.forward): every: all the tokens' (True), or those of
    the step's rows it names (int32, on the device)."""
    rows, seen, _ = llama.around(w, c, places, caches.size, slots, length)
    at = SimpleNamespace(places=places, rows=rows, seen=seen, chunk=not slots and places.cols > 1, dead=caches.size // slots - 1 if slots else -1)
    x = w["embed"].gather(ids).cast("fp32")
    blocks = w.get("_blocks") or [llama.block(w, f"l{l}.") for l in range(c.layers)]
    for b, p, cache in zip(c.blocks, blocks, caches):
        x = layer(x, p, b, c, at, cache)
    h = mixers.dyt(x, w, "final.norm").cast(c.dtype)
    if isinstance(every, Tensor):
        h = h.realize().gather(every)
    elif not (slots or every):
        h = h.realize()[:, x.rows - 1:, :]
    return h.matmul(w["head"], dtype="fp32")


def kv_cache(c, size, zeros, slots=1):
    make = lambda shape, dtype=c.dtype: zeros(shape, dtype)
    return mixers.Caches(size, [MIXERS[b.type][1](b.mixer, size, make, slots) for b in c.blocks])


def slot(c, caches, u, slots):
    """Sequence u's part of caches made for several, in place."""
    part = caches.size // slots
    return mixers.Caches(part, [x[:, u * part:(u + 1) * part, :] if x.rows == caches.size and x.batch == 1 and b.type == "latent_attention" else x[u:u + 1, :, :]
                         for x, b in zip(caches, c.blocks)])


def random_weights(rt, c, prec=None, seed=0, scale=0.02):
    """Random weights in c's shapes made on the device: matrices N(0, scale), norms 1, slopes and biases small."""
    gen = torch.Generator(device=rt.device).manual_seed(seed)

    def matrix(name, n, k, batch=1, f=None):  # [k, n], each output column's weights together
        x = torch.empty(batch, n, k, dtype=torch.float32, device=rt.device).normal_(0, scale, generator=gen).bfloat16()
        t = Tensor(rt, n, k, batch=batch, buf=x)
        f = weight_format(name, prec)
        w[name] = t.T if f == "bf16" else t.T.cast(f).realize()

    def vector(name, n, value=1.0):
        w[name] = Tensor.of(rt, np.full((1, n), value, np.float32), "fp32")

    def norm(name):
        vector(name, c.dim), vector(name + ".b", c.dim, 0.0), vector(name + ".alpha", 1, 0.5)

    w = {}
    for l, b in enumerate(c.blocks):
        pre, m, d = f"l{l}.", b.mixer, c.dim
        norm(pre + "norm1"), norm(pre + "norm1b")
        if b.type == "latent_attention":
            matrix(pre + "mix.in", m.q_rank + m.kv_rank + m.rot_dim + m.heads, d)
            vector(pre + "mix.dq.norm", m.q_rank), vector(pre + "mix.dkv.norm", m.kv_rank), vector(pre + "mix.sink", m.heads, 0.0)
            matrix(pre + "mix.uq", m.heads * (m.dim + m.rot_dim), m.q_rank)
            matrix(pre + "mix.uk", m.kv_rank, m.dim, m.heads), matrix(pre + "mix.uv", m.vdim, m.kv_rank, m.heads)
        else:
            matrix(pre + "mix.qkvg", m.heads * 2 * (m.dim + m.vdim), d), vector(pre + "mix.norm", m.heads * m.vdim)
        matrix(pre + "mix.o", d, m.heads * m.vdim)
        if b.mlp:
            norm(pre + "norm2"), norm(pre + "norm2b")
            matrix(pre + "mlp.gate_up", 2 * b.mlp.ff, d), matrix(pre + "mlp.down", d, b.mlp.ff)
    norm("final.norm")
    matrix("head", c.vocab, c.dim)
    embed = torch.empty(c.vocab, c.dim, dtype=torch.float32, device=rt.device).normal_(0, 1, generator=gen)
    w["embed"] = Tensor(rt, c.vocab, c.dim, dtype=c.dtype, buf=embed.to(torch.float32 if c.dtype == "fp32" else torch.bfloat16).view(1, c.vocab, c.dim))
    llama.settle(rt, w)
    w["_blocks"] = [llama.block(w, f"l{l}.") for l in range(c.layers)]
    return w
