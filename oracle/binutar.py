"""TEST INFRASTRUCTURE (not the product): the Binutar decoder as plain numpy in float64, one function per mechanism,
token by token where the design is a recurrence and key by key where it is attention.  Weights are {name: array} under
the checkpoint's own tensor names (linear weights [out, in]); the configuration is the parsed config.json."""
import math

import numpy as np

f64 = np.float64


def sigmoid(x):
    return 1 / (1 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def rms(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def dyt(x, w, name):
    """Dynamic Tanh: a scalar slope, then a weight and a bias per column."""
    return np.tanh(f64(w[name + ".alpha"].reshape(())) * x) * w[name] + w[name + ".b"]


def yarn(rot):
    """(frequencies of the pairs, factor of cos and sin) of a rotation: plain, or with YaRN's ramp between the frequencies
    that turn often enough within the original context (kept) and those that do not (divided)."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([f64(base) ** (-2 * i / dims) for i in range(dims // 2)])
    if not s:
        return f, 1.0
    dim = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(s["fast"])), 0), min(math.ceil(dim(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0, 1)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1


def rotate(x, places, rot):
    """The first rot.dims of x's last axis turned by each token's angle, neighbours a pair; the rest as it is."""
    f, mag = yarn(rot)
    dims, out = rot["dims"], np.array(x, f64)
    for t, p in enumerate(places):
        for i in range(dims // 2):
            c, s = math.cos(p * f[i]) * mag, math.sin(p * f[i]) * mag
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i], out[t, ..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def attend(q, k, v, places, key_places, scale, sink):
    """q [T, H, D], k [L, H, D], v [L, H, V]: causal softmax by places; the sink is one more term of the denominator."""
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]))
    for t, p in enumerate(places):
        seen = np.asarray(key_places) <= p
        for h in range(q.shape[1]):
            s = k[seen, h] @ q[t, h] * scale
            m = max(s.max(), sink[h])
            e = np.exp(s - m)
            out[t, h] = (e[:, None] * v[seen, h]).sum(0) / (e.sum() + math.exp(sink[h] - m))
    return out


def latent_attention(h, w, pre, m, eps, places, cache):
    """cache: a dict this layer keeps for the sequence: the latents, the rotated key parts and their places."""
    H, dim, rd, vd, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    cq = rms(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).reshape(T, H, dim + rd)
    down = h @ w[pre + "dkv"].T
    c, kr = rms(down[:, :rank], w[pre + "dkv.norm"], eps), rotate(down[:, rank:], places, m["rot"])
    for name, x in (("c", c), ("kr", kr)):
        cache[name] = np.concatenate([cache[name], x]) if name in cache else x
    cache["p"] = list(cache.get("p", [])) + list(places)
    L = len(cache["p"])
    k = np.concatenate([(cache["c"] @ w[pre + "uk"].T).reshape(L, H, dim), np.repeat(cache["kr"][:, None], H, 1)], 2)
    v = (cache["c"] @ w[pre + "uv"].T).reshape(L, H, vd)
    q = np.concatenate([q[:, :, :dim], rotate(q[:, :, dim:], places, m["rot"])], 2)
    o = attend(q, k, v, places, cache["p"], m["scale"], w[pre + "sink"])
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * vd) @ w[pre + "o"].T


def recurrence(q, k, v, decay, state):
    """q, k [T, H, D], v [T, H, V], state [H, D, V] (changed in place): S = decay S + k v^T, then o = S^T q."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            state[h] = decay[h] * state[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = state[h].T @ q[t, h]
    return out


def lightning(h, w, pre, m, eps, cache):
    H, dim, vd, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(h @ w[pre + n].T).reshape(T, H, -1) for n in "qkv")
    state = cache.setdefault("s", np.zeros((H, dim, vd)))
    o = recurrence(q, k, v, m["decay"], state).reshape(T, H * vd)
    return (rms(o, w[pre + "norm"], eps) * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def feed_forward(h, w, pre, m):
    return glu(h @ w[pre + "gate"].T, h @ w[pre + "up"].T, m["limit"]) @ w[pre + "down"].T


def layer(x, w, i, entry, eps, places, cache):
    pre = f"l{i}."
    h = dyt(x, w, pre + "norm1")
    if entry["type"] == "latent_attention":
        y = latent_attention(h, w, pre + "mix.", entry["mixer"], eps, places, cache)
    else:
        y = lightning(h, w, pre + "mix.", entry["mixer"], eps, cache)
    x = x + dyt(y, w, pre + "norm1b")
    if entry.get("mlp"):
        x = x + dyt(feed_forward(dyt(x, w, pre + "norm2"), w, pre + "mlp.", entry["mlp"]), w, pre + "norm2b")
    return x


def forward(ids, first, w, cfg, caches, residuals=None):
    """Logits of every token of ids, at places first.., one sequence; caches: a list of dicts, one a layer (start with
    empty ones).  residuals: a list that receives the residual stream after every layer."""
    places = list(range(first, first + len(ids)))
    x = f64(w["embed"])[list(ids)]
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, w, i, entry, cfg["norm"]["eps"], places, caches[i])
        if residuals is not None:
            residuals.append(x)
    return dyt(x, w, "final.norm") @ w["head"].T


def caches(cfg):
    return [{} for _ in cfg["layers"]]


def tensors(cfg):
    """{name: shape} of a configuration's checkpoint."""
    d, out = cfg["width"], {"embed": [cfg["vocab"], cfg["width"]], "head": [cfg["vocab"], cfg["width"]]}

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = [d], [d], []
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        norm(p + "norm1"), norm(p + "norm1b")
        H = m["heads"]
        if e["type"] == "latent_attention":
            out |= {p + "mix.dq": [m["q_rank"], d], p + "mix.dq.norm": [m["q_rank"]], p + "mix.uq": [H * (m["dim"] + m["rot_dim"]), m["q_rank"]],
                    p + "mix.dkv": [m["kv_rank"] + m["rot_dim"], d], p + "mix.dkv.norm": [m["kv_rank"]], p + "mix.uk": [H * m["dim"], m["kv_rank"]],
                    p + "mix.uv": [H * m["vdim"], m["kv_rank"]], p + "mix.sink": [H], p + "mix.g": [H, d], p + "mix.o": [d, H * m["vdim"]]}
        else:
            out |= {p + "mix.q": [H * m["dim"], d], p + "mix.k": [H * m["dim"], d], p + "mix.v": [H * m["vdim"], d], p + "mix.g": [H * m["vdim"], d],
                    p + "mix.o": [d, H * m["vdim"]], p + "mix.norm": [H * m["vdim"]]}
        if e.get("mlp"):
            norm(p + "norm2"), norm(p + "norm2b")
            f = e["mlp"]["ff"]
            out |= {p + "mlp.gate": [f, d], p + "mlp.up": [f, d], p + "mlp.down": [d, f]}
    norm("final.norm")
    return out
