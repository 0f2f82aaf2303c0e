"""Layer parts beside the Llama block's (llama.attention, llama.mlp, llama.rms): token mixers that keep something per
sequence - attention over cached latents, linear attention with a decaying state - a norm and a gated unit.  Every
constant is a parameter; a design's module (binutar.py) says which parts it is made of.

A mixer is a pair of functions: `*_cache(m, size, zeros, slots)` makes what it keeps for `slots` sequences of size / slots
places each, and the mixer itself maps normed rows to rows, given its weights, its sizes m and where the tokens stand
(at: places, cache rows, and what llama.around says they see)."""
import math

import torch

from .tensor import Tensor


def dyt(x, p, name):
    """Dynamic Tanh in the place of a norm: tanh(alpha x) w + b, alpha a scalar."""
    return (x * p[name + ".alpha"]).tanh() * p[name] + p[name + ".b"]


def clamped_glu(gate, up, limit, slope):
    """g sigmoid(slope g) (u + 1) with the gate's half cut at limit and the other within -limit .. limit."""
    g, u = gate.minimum(limit), up.maximum(-limit).minimum(limit)
    return g * (g * slope).sigmoid() * (u + 1)


def clamped_mlp(h, p, pre, limit, slope):
    """down(clamped_glu(gate(h), up(h))), gate and up side by side in gate_up."""
    gate_up = h.matmul(p[pre + "gate_up"], dtype="fp32")
    m = gate_up.cols // 2
    return clamped_glu(gate_up[:, :m], gate_up[:, m:], limit, slope).cast(h.dtype).matmul(p[pre + "down"], dtype="fp32")


# -------------------------------------------------------------------- rotation

def frequencies(rot):
    """A rotation's frequencies (a number a pair, in double) and the factor of its cos and sin: plain powers of the base,
    or YaRN's: pairs that turn more than `fast` times within the original context keep theirs, those that turn less than
    `slow` times have it divided, with a ramp in between."""
    f = [rot.base ** (-2.0 * i / rot.dims) for i in range(rot.dims // 2)]
    s = rot.scaling
    if not s:
        return f, 1.0
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
    p: in (query latent | key-value latent | key part | gates, as far as the design has them), uq, uk and uv by head, o."""
    H, rank, rd, rt = m.heads, m.kv_rank, m.rot_dim, h.rt
    turn = rotation(rt, m.rot)
    base, last, length, _ = at.seen
    down = h.matmul(p["mix.in"], dtype="fp32").realize()
    c_q = down.latent_put(turn, at.places, at.rows, cache, m.q_rank, p["mix.dq.norm"], p["mix.dkv.norm"], eps)
    q = c_q.matmul(p["mix.uq"], dtype=h.dtype).split(H)
    query = Tensor(rt, h.rows, H * (rank + rd), dtype=h.dtype)
    by_head = query.split(H)
    q[:, :, :m.dim].matmul(p["mix.uk"]).realize(into=by_head[:, :, :rank])
    q[:, :, m.dim:].rotate_pairs(turn, at.places, into=by_head[:, :, rank:])
    o = query.attend_latent(cache, base, last, rank, m.scale, p.get("mix.sink"), length, chunk=at.chunk)
    values = Tensor(rt, h.rows, H * m.vdim, dtype=h.dtype)
    gates = down[:, :, down.cols - H:].permute(2, 1, 0)  # a number a head and token
    (o.split(H).matmul(p["mix.uv"]) * gates.sigmoid()).cast(h.dtype).realize(into=values.split(H))
    return values.matmul(p["mix.o"], dtype="fp32")


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
