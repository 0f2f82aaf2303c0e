"""Layer parts beside the Llama block's (llama.attention, llama.mlp, llama.rms): token mixers that keep something per
sequence, feed-forwards, a norm.  Every constant is a parameter; a design's module (binutar.py, labepel.py, vunadra.py, ronavik.py) says
which parts it is made of.

They are: attention over cached latents, grouped-query attention within spans or windows of the sequence, with or without a
rotation and a short convolution, or weighted by sigmoids, linear attention with a decaying state, a state space whose decay is a token's
own, a gated linear recurrence, and that beside attention; a clamped, a SiLU- and a GELU-gated unit, a mixture of experts; Dynamic Tanh.

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


def slot(caches, u, slots):
    """Sequence u's part of caches made for several, in place: of cached rows its run, of states (what follows the rows in a tuple; None stands
    for no rows) its own."""
    part = caches.size // slots
    rows = lambda x: None if x is None else x[:, u * part:(u + 1) * part, :]
    return Caches(part, [(rows(x[0]), *(s[u:u + 1, :, :] for s in x[1:])) if isinstance(x, tuple) else rows(x) for x in caches])


def project(h, w):
    """h @ w in fp32, its rows whole 16-byte pieces apart whatever w's width: parts of them are read four columns at a time."""
    out = Tensor(h.rt, h.rows, -(-w.cols // 8) * 8, dtype="fp32")[:, :, :w.cols]
    return h.matmul(w, dtype="fp32").realize(into=out)


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


def mixture(h, logits, p, pre, k, scored=False, identity=0, scale=1.0, clamp=None, as_scored=False, on_input=False):
    """A mixture of experts for rows h with their router logits (fp32): the k largest of each row's, weighted by their softmax.
    p: gate_up and down as batches of experts, the router's bias if it has one (router.b), a shared expert's own pair
    (shared.gate_up, shared.down) if there is one.  scored: the softmax of all logits ("sigmoid": each one's own sigmoid), with the bias,
    chooses, and without it weighs, over the chosen ones' sum unless as_scored; on_input: a weight is on its expert's input; experts with an `up` instead of gate_up have
    the unit max(up, 0)^2; identity: the router's last so many outputs stand for experts that give back their input; scale: of the weights; clamp:
    the experts' units are clamped ones (limit, slope).  Returns (the shared expert's result or None, (the chosen experts' rows,
    their routes)) as Tensor.add_norm adds them up."""
    relu2 = pre + "up" in p
    gate_up, down = p[pre + ("up" if relu2 else "gate_up")], p[pre + "down"]
    routes = logits.route(gate_up.batch + identity, k, p.get(pre + "router.b"), scored, identity, scale, as_scored, on_input)
    shared = gated_mlp(h, p, pre + "shared.") if pre + "shared.gate_up" in p else None
    if gate_up.dtype not in BFP:
        return shared, (h.experts(routes, gate_up, down, clamp, relu2), routes)
    assert not (identity or clamp or relu2 or on_input), "block-float experts are plain ones"
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


def sigmoid_width(m):
    """Columns of the joint projection: queries, keys, values."""
    return (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim


def sigmoid_attention(joint, p, m, eps, at, cache, scale=1.0, into=None):
    """Attention without a softmax: a key's weight is the sigmoid of its score and a number of the head (mix.pb).  joint: q | k | v, fp32; p: the heads'
    norms (mix.q.norm, mix.k.norm); queries by the temperature of their place (m.q_temp).  The heads side by side times scale (into: there)."""
    base, last, length, _ = at.seen
    q = joint.heads_put(m.heads, m.dim, m.vdim, at.rows, cache, None, p["mix.q.norm"], p["mix.k.norm"], eps, places=at.places, temperature=m.q_temp and (m.q_temp.coef, m.q_temp.every))
    return q.attend_heads(cache, base, last, m.vdim, m.scale, length, chunk=at.chunk, key_bias=p["mix.pb"], out_scale=scale, into=into)


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


# -------------------------------------------------------------------- a state space whose decay is a token's own

def state_space_width(m):
    """Columns of the joint projection: a gate and values (heads x vdim each), keys and queries (groups x state each), step sizes (heads)."""
    return 2 * m.heads * m.vdim + 2 * m.groups * m.state + m.heads


def state_space_cache(m, size, zeros, slots):
    """No rows; what the convolution needs of earlier tokens, and a [state, vdim] matrix a head, fp32."""
    return None, zeros((slots, max(m.conv - 1, 1), m.heads * m.vdim + 2 * m.groups * m.state), "fp32"), zeros((slots, m.heads * m.state, m.vdim), "fp32")


def state_space(joint, p, m, eps, at, cache):
    """joint: z | x | B | C | dt, fp32.  x, B and C through a short convolution and SiLU, the recurrence, the values beside it (mix.D), SiLU of z, RMSNorm in
    m.norm_groups parts.  p: mix.conv, mix.conv.b, mix.dt_bias, mix.A_log, mix.D, mix.norm, mix.o."""
    _, conv, state = cache
    inner = m.heads * m.vdim
    n = 2 * inner + 2 * m.groups * m.state
    dtype = at.dtype
    xbc = joint[:, :, inner:n].short_conv(p["mix.conv"], at.places, conv, at.dead, bias=p["mix.conv.b"], silu=True, dtype=dtype)
    y = xbc.selective_scan(m.heads, m.groups, m.state, m.vdim, joint[:, :, n:n + m.heads], p["mix.dt_bias"], p["mix.A_log"], p["mix.D"], at.places, state, at.dead)
    return y.gated_rms(joint[:, :, :inner], p["mix.norm"], eps, before=True, parts=m.norm_groups, dtype=dtype).matmul(p["mix.o"], dtype=dtype)


# -------------------------------------------------------------------- a gated linear recurrence, and that beside attention

LRU_RATE = -8.0  # log of the decay: this times a gate times the softplus of a number a column


def recurrent_cache(m, size, zeros, slots):
    """No rows; what the convolution needs of earlier tokens, and a number a column, fp32."""
    return None, zeros((slots, max(m.conv - 1, 1), m.width), "fp32"), zeros((slots, 1, m.width), "fp32")


def recurrent_block(joint, p, m, at, cache, scale=1.0, into=None):
    """joint: y | x, fp32.  x through a short convolution, a gated linear recurrence whose gates are m.blocks matrices of their own (mix.gates: each block's
    r | i), times the GELU of y.  p: mix.y.b, mix.x.b, mix.conv, mix.conv.b, mix.gates, mix.gates.b, mix.lam.  The result times scale (into: there)."""
    _, conv, state = cache
    u = joint[:, :, m.width:2 * m.width].short_conv(p["mix.conv"], at.places, conv, at.dead, bias=p["mix.conv.b"], in_bias=p["mix.x.b"], dtype=at.dtype)
    gates = Tensor(joint.rt, joint.rows, 2 * m.width, dtype="fp32")
    u.split(m.blocks).matmul(p["mix.gates"], dtype="fp32").realize(into=gates.split(m.blocks))
    return u.lru_scan(gates, joint[:, :, :m.width], p["mix.lam"], LRU_RATE, m.blocks, at.places, state, at.dead, p["mix.gates.b"], p["mix.y.b"], scale, into)


def parallel_width(m):
    return sigmoid_width(m.left) + 2 * m.right.width


def parallel_cache(m, size, zeros, slots):
    return (heads_cache(m.left, size, zeros, slots), *recurrent_cache(m.right, size, zeros, slots)[1:])


def parallel(joint, p, m, eps, at, cache):
    """Attention and a recurrent block that read the same rows, each by a scale of its own.  joint: q | k | v | y | x, fp32; their output matrices are one
    (mix.o), the attention's rows above the block's."""
    n, wide = sigmoid_width(m.left), m.left.heads * m.left.vdim
    both = Tensor(joint.rt, joint.rows, wide + m.right.width, dtype=at.dtype)
    sigmoid_attention(joint[:, :, :n], p, m.left, eps, at, cache[0], m.left_scale, both[:, :, :wide])
    recurrent_block(joint[:, :, n:], p, m.right, at, cache, m.right_scale, both[:, :, wide:])
    return both.matmul(p["mix.o"], dtype=at.dtype)
