"""Layer parts beside the Llama block's (llama.attention, llama.mlp, llama.rms): token mixers that keep something per
sequence, feed-forwards, a norm.  Every constant is a parameter; a design's module (binutar.py, labepel.py, vunadra.py) says which parts
it is made of.

They are: attention over cached latents, grouped-query attention within spans or windows of the sequence, with or without a
rotation and a short convolution, linear attention with a decaying state; a clamped, a SiLU- and a GELU-gated unit, a mixture of
experts; Dynamic Tanh.

A mixer is a pair of functions: `*_cache(m, size, zeros, slots)` makes what it keeps for `slots` sequences of size / slots
places each, and the mixer itself maps normed rows to rows, given its weights, its sizes m and where the tokens stand
(at: places, cache rows, and what llama.around says they see)."""
import math

import torch

from . import llama
from .tensor import BFP, Tensor, clamped_glu


class Caches(list):
    """A layer's cache or state each, for sequences that share `size` places."""

    def __init__(self, size, caches):
        super().__init__(caches)
        self.size = size


def dyt(x, p, name):
    """Dynamic Tanh in the place of a norm: tanh(alpha x) w + b, alpha a scalar."""
    return (x * p[name + ".alpha"]).tanh() * p[name] + p[name + ".b"]


def clamped_mlp(h, p, pre, limit, slope):
    """down(clamped_glu(gate(h), up(h))), gate and up side by side in gate_up."""
    gate_up = h.matmul(p[pre + "gate_up"], dtype="fp32")
    m = gate_up.cols // 2
    return clamped_glu(gate_up[:, :m], gate_up[:, m:], limit, slope).cast(h.dtype).matmul(p[pre + "down"], dtype="fp32")


def gated_mlp(h, p, pre):
    """down(silu(gate(h)) * up(h)), gate and up side by side in gate_up."""
    gate_up = p[pre + "gate_up"]
    both = h.matmul(gate_up, dtype="bf16" if gate_up.dtype in BFP else "fp32")
    m = gate_up.cols // 2
    return llama.glu(both[:, :m], both[:, m:]).cast(h.dtype).matmul(p[pre + "down"], dtype=h.dtype)


def gelu_mlp(h, p, pre):
    """down(gelu(gate(h)) * up(h)), gate and up side by side in gate_up, their biases in gate_up.b; down's is left to what adds it."""
    unit = h.matmul(p[pre + "gate_up"], dtype="fp32").gelu_gated(p.get(pre + "gate_up.b"), h.dtype)
    return unit.matmul(p[pre + "down"], dtype=h.dtype)


def mixture(h, logits, p, pre, k, scored=False, identity=0, scale=1.0, clamp=None):
    """A mixture of experts for rows h with their router logits (fp32): the k largest of each row's, weighted by their softmax.
    p: gate_up and down as batches of experts, the router's bias if it has one (router.b), a shared expert's own pair
    (shared.gate_up, shared.down) if there is one.  scored: the softmax of all logits, with the bias, chooses, and without it
    weighs; identity: the router's last so many outputs stand for experts that give back their input; scale: of the weights; clamp:
    the experts' units are clamped ones (limit, slope).  Returns (the shared expert's result or None, (the chosen experts' rows,
    their routes)) as Tensor.add_norm adds them up."""
    gate_up, down = p[pre + "gate_up"], p[pre + "down"]
    routes = logits.route(gate_up.batch + identity, k, p.get(pre + "router.b"), scored, identity, scale)
    shared = gated_mlp(h, p, pre + "shared.") if pre + "shared.gate_up" in p else None
    if gate_up.dtype not in BFP:
        return shared, (h.experts(routes, gate_up, down, clamp), routes)
    assert not (identity or clamp), "block-float experts are plain ones"
    of = lambda buf, dtype: Tensor(h.rt, routes.T, routes.k, dtype=dtype, buf=buf.view(1, routes.T, routes.k))
    y = llama.experts(h, {"experts.gate_up": gate_up, "experts.down": down}, of(routes.ids, "int32"), of(routes.weights, "fp32"))
    return (y if shared is None else shared + y), None


# -------------------------------------------------------------------- rotation

def frequencies(rot):
    """A rotation's frequencies (a number a pair, in double) and the factor of its cos and sin: plain powers of the base;
    YaRN's (a scaling with `fast` and `slow`): pairs that turn more than `fast` times within the original context keep theirs, those
    that turn less than `slow` times have it divided, with a ramp in between; or Llama 3.1's (`high` and `low`): waves of less than
    1 / high of the original context keep theirs, those of more than 1 / low have it divided, with a blend in between."""
    f = [rot.base ** (-2.0 * i / rot.dims) for i in range(rot.dims // 2)]
    s = rot.scaling
    if not s:
        return f, 1.0
    if hasattr(s, "high"):
        part = lambda v: min(max((s.original * v / (2 * math.pi) - s.low) / (s.high - s.low), 0.0), 1.0)  # 1: kept, 0: divided
        return [(1 - part(v)) * v / s.factor + part(v) * v for v in f], 1.0
    pair = lambda turns: rot.dims * math.log(s.original / (2 * math.pi * turns)) / (2 * math.log(rot.base))
    lo, hi = max(math.floor(pair(s.fast)), 0), min(math.ceil(pair(s.slow)), rot.dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
    return [a / s.factor * r + a * (1 - r) for a, r in zip(f, ramp)], 0.1 * math.log(s.factor) + 1


def rotation(rt, rot):
    """(frequencies on the device, columns that turn, factor): a constant of the program, made once."""
    s = rot.scaling
    key = ("rotation", rot.base, rot.dims, tuple(sorted(vars(s).items())) if s else None)
    if key not in rt.numbers:
        f, mag = frequencies(rot)
        rt.numbers[key] = (torch.tensor(f or [0.0], dtype=torch.float64, device=rt.device), rot.dims, mag)
    return rt.numbers[key]


# -------------------------------------------------------------------- attention over latents

def latent_cache(m, size, zeros, slots):
    """A row a place: the latent and the turned key part, shared by all heads."""
    return zeros((1, size, m.kv_rank + m.rot_dim))


def latent_attention(h, p, m, eps, at, cache):
    """Attention whose keys and values are made from a cached latent.  A head's key is W_uk c and its value W_uv c; here the
    query goes through W_uk instead and the weighted latents through W_uv, so that the cache is read as it is.
    p: in (query latent, or the queries themselves where the design has none | key-value latent | key part | a gate per head, if the
    design has them), uq, uk and uv by head, o.  m.window: a token sees the last so many places."""
    H, rank, rd, rt, q_rank = m.heads, m.kv_rank, m.rot_dim, h.rt, getattr(m, "q_rank", 0)
    turn = rotation(rt, m.rot)
    base, last, length, _ = at.seen
    down = h.matmul(p["mix.in"], dtype="fp32").realize()
    query = Tensor(rt, h.rows, H * (rank + rd), dtype=h.dtype)
    by_head = query.split(H)
    if q_rank:
        c_q = down.latent_put(turn, at.places, at.rows, cache, q_rank, p["mix.dq.norm"], p["mix.dkv.norm"], eps)
        q = c_q.matmul(p["mix.uq"], dtype=h.dtype).split(H)
        q[:, :, m.dim:].rotate_pairs(turn, at.places, into=by_head[:, :, rank:])
        plain = q[:, :, :m.dim]
    else:
        plain = down.latent_heads_put(turn, at.places, at.rows, cache, H, m.dim, by_head[:, :, rank:], p["mix.dkv.norm"], eps).split(H)
    plain.matmul(p["mix.uk"]).realize(into=by_head[:, :, :rank])
    o = query.attend_latent(cache, base, last, rank, m.scale, p.get("mix.sink"), length, chunk=at.chunk, window=getattr(m, "window", 0))
    values = Tensor(rt, h.rows, H * m.vdim, dtype=h.dtype)
    used = (q_rank or H * (m.dim + rd)) + rank + rd
    if down.cols == used:
        o.split(H).matmul(p["mix.uv"]).realize(into=values.split(H))
    else:
        gates = down[:, :, used:].permute(2, 1, 0)  # a number a head and token
        (o.split(H).matmul(p["mix.uv"]) * gates.sigmoid()).cast(h.dtype).realize(into=values.split(H))
    return values.matmul(p["mix.o"], dtype="fp32")


# -------------------------------------------------------------------- grouped-query attention

def heads_width(m):
    """Columns of the joint projection: queries, keys, values, and a gate for each column of the result."""
    return (m.heads + m.kv_heads) * m.dim + (m.kv_heads + m.heads) * m.vdim


def heads_cache(m, size, zeros, slots):
    """A key and its value side by side, a row a place and key head."""
    return zeros((m.kv_heads, size, m.dim + m.vdim))


def heads_attention(joint, p, m, eps, at, cache, sink=None):
    """Attention of query heads that share key heads, each token within its own span of m.mask.size places.
    joint: q | k | v | gate (| more), fp32; p: their biases side by side (mix.b), the heads' norms (mix.q.norm, mix.k.norm), the
    output's matrix (mix.o); with m.v_mix, the values of the first such layer of the pass (at.first) are mixed in by mix.vmix.
    sink: a number that joins every head's denominator as exp(sink)."""
    H, n, wide = m.heads, (m.heads + m.kv_heads) * m.dim, m.kv_heads * m.vdim
    base, last, length, _ = at.seen
    mix = None
    if m.v_mix:
        mix = (*at.first, p["mix.vmix"]) if at.first else None
        at.first = at.first or (joint[:, n:n + wide], p["mix.b"][:, n:])
    q = joint.heads_put(H, m.dim, m.vdim, at.rows, cache, p["mix.b"], p["mix.q.norm"], p["mix.k.norm"], eps, mix)
    key = ("sink", H, sink)
    if sink is not None and key not in joint.rt.numbers:
        joint.rt.numbers[key] = Tensor.of(joint.rt, [[sink] * H], "fp32")
    gate = joint[:, n + wide:n + wide + H * m.vdim]
    o = q.attend_heads(cache, base, last, m.vdim, m.scale, length, m.mask.size, joint.rt.numbers.get(key), gate, chunk=at.chunk)
    return o.matmul(p["mix.o"], dtype=o.dtype)


def turned_width(m):
    """Columns of the joint projection: queries, keys and, where they are not the keys, values."""
    return (m.heads + m.kv_heads) * m.dim + (0 if m.keys_are_values else m.kv_heads * m.vdim)


def turned_cache(m, size, zeros, slots):
    """heads_cache, and, with a short convolution (m.conv taps), what it needs of earlier tokens: (rows, state)."""
    rows = heads_cache(m, size, zeros, slots)
    return (rows, zeros((slots, max(m.conv - 1, 1), turned_width(m)), "fp32")) if m.conv else rows


def turned_attention(h, p, m, eps, at, cache):
    """Attention of turned query heads that share turned key heads, each token seeing all before it or the last m.window places;
    m.softcap caps the scores (0: it does not).  p: in (q | k | v; with m.keys_are_values q | k), what the projection's columns go
    through - biases (mix.b), a short convolution (mix.conv, [m.conv taps, columns]), norms (mix.q.norm, mix.k.norm; m.norm_all:
    over all heads together) -, the output's matrix (mix.o; its bias is left to what adds the result)."""
    rows, state = cache if m.conv else (cache, None)
    base, last, length, _ = at.seen
    joint = h.matmul(p["mix.in"], dtype="fp32").realize()
    q = joint.heads_put(m.heads, m.dim, m.vdim, at.rows, rows, p.get("mix.b"), p.get("mix.q.norm"), p.get("mix.k.norm"), eps, norm_all=m.norm_all, keys_are_values=m.keys_are_values,
                        rotation=rotation(h.rt, m.rot), places=at.places, conv=p.get("mix.conv"), state=state, dead=at.dead)
    o = q.attend_heads(rows, base, last, m.vdim, m.scale, length, chunk=at.chunk, window=m.window, softcap=m.softcap)
    return o.matmul(p["mix.o"], dtype=o.dtype)


# -------------------------------------------------------------------- linear attention with a decaying state

def decay_cache(m, size, zeros, slots):
    """A [dim, vdim] matrix a head and sequence, fp32."""
    return zeros((slots, m.heads * m.dim, m.vdim), "fp32")


def decay_attention(h, p, m, eps, at, state):
    """q, k and v through SiLU, the recurrence, RMSNorm over all heads together, a sigmoid gate.  p: qkvg side by side."""
    H = m.heads
    n = H * (2 * m.dim + m.vdim)
    key = ("decay", tuple(m.decay))
    if key not in h.rt.numbers:
        h.rt.numbers[key] = Tensor.of(h.rt, [list(m.decay)], "fp32")
    qkvg = h.matmul(p["mix.qkvg"], dtype=h.dtype).silu_columns(n).realize()
    o = qkvg.decay_scan(H, m.dim, m.vdim, h.rt.numbers[key], at.places, state, at.dead)
    return o.gated_rms(qkvg[:, :, n:], p["mix.norm"], eps).matmul(p["mix.o"], dtype="fp32")
