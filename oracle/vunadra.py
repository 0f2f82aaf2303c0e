"""TEST INFRASTRUCTURE (not the product): the Vunadra decoder as plain numpy in float64, one function per mechanism, query by
query and expert by expert.  Weights are {name: array} under the checkpoint's own tensor names (linear weights [out, in]); the
configuration is the parsed config.json."""
import math

import numpy as np

f64 = np.float64
SLOPE = 1.702  # of an expert's gate


def sigmoid(x):
    return 1 / (1 + np.exp(-x))


def rms(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def gelu(z):
    return 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def linear(h, w, name):
    """W h, and the bias where the checkpoint has one."""
    y = h @ f64(w[name]).T
    return y + w[name + ".b"] if name + ".b" in w else y


# ---- rotation

def yarn(f, rot):
    """Pairs that turn often within the original context keep their frequency, those that turn seldom have it divided."""
    s, dims = rot["scaling"], rot["dims"]
    where = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(len(f)) - lo) / max(hi - lo, 0.001), 0, 1)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1


def by_wavelength(f, rot):
    """Short waves keep their frequency, long ones have it divided, with a blend between the two bounds."""
    s = rot["scaling"]
    out = []
    for v in f:
        wave = 2 * math.pi / v
        if wave < s["original"] / s["high"]:
            out.append(v)
        elif wave > s["original"] / s["low"]:
            out.append(v / s["factor"])
        else:
            blend = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - blend) * v / s["factor"] + blend * v)
    return np.array(out), 1.0


def frequencies(rot):
    f = rot["base"] ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    if not rot.get("scaling"):
        return f, 1.0
    return yarn(f, rot) if "fast" in rot["scaling"] else by_wavelength(f, rot)


def rotate(x, places, rot):
    """x [T, heads, width]: the columns (2i, 2i + 1) of the first rot.dims turned by their token's place."""
    f, mag = frequencies(rot)
    a = f64(places)[:, None, None] * f
    c, s = np.cos(a) * mag, np.sin(a) * mag
    out = x.copy()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2], out[..., 1:rot["dims"]:2] = u * c - v * s, v * c + u * s
    return out


# ---- attention

def window_start(place, size):
    """The first place that a token sees through a window of `size` places (None: all before it)."""
    return max(0, place - size + 1) if size else 0


def capped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def attend(q, k, v, places, scale, size=None, cap=None):
    """q [T, H, D] at places over k [L, G, D], v [L, G, V] of the places 0..L-1; a key head serves H / G query heads in a row."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t, p in enumerate(places):
        seen = slice(window_start(p, size), p + 1)
        for h in range(H):
            s = capped(k[seen, h // rep] @ q[t, h] * scale, cap)
            e = np.exp(s - s.max())
            out[t, h] = e @ v[seen, h // rep] / e.sum()
    return out


def keep(cache, **new):
    """What a layer keeps of a sequence, with the new tokens' added; returned in the order given."""
    for name, x in new.items():
        cache[name] = np.concatenate([cache[name], x]) if name in cache else x
    return [cache[name] for name in new]


def convolved(u, kernel, before):
    """y_t = sum_j kernel[:, j] u_(t - taps + 1 + j); before: the last taps - 1 rows of earlier tokens, or zeros."""
    taps = kernel.shape[1]
    rows = np.concatenate([before, u])
    return sum(kernel[:, j] * rows[j:j + len(u)] for j in range(taps)), rows[len(rows) - (taps - 1):]


def short_convolution(h, w, name, cache):
    kernel = f64(w[name + ".conv"])
    u = linear(h, w, name)
    y, cache[name] = convolved(u, kernel, cache.get(name, np.zeros((kernel.shape[1] - 1, u.shape[1]))))
    return y


def attention(h, w, pre, m, eps, places, cache):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q, k, v = (short_convolution(h, w, pre + n, cache) for n in "qkv")
    q, k = rotate(q.reshape(T, H, m["dim"]), places, m["rot"]), rotate(k.reshape(T, G, m["dim"]), places, m["rot"])
    keys, values = keep(cache, keys=k, values=v.reshape(T, G, m["vdim"]))
    return linear(attend(q, keys, values, places, m["scale"]).reshape(T, -1), w, pre + "o")


def attention_2(h, w, pre, m, eps, places, cache):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q, k = linear(h, w, pre + "q"), linear(h, w, pre + "k")
    v = k.reshape(T, G, m["dim"])
    q = rotate(rms(q, w[pre + "q.norm"], eps).reshape(T, H, m["dim"]), places, m["rot"])
    k = rotate(rms(k, w[pre + "k.norm"], eps).reshape(T, G, m["dim"]), places, m["rot"])
    keys, values = keep(cache, keys=k, values=v)
    return linear(attend(q, keys, values, places, m["scale"], m["mask"]["size"], m["softcap"]).reshape(T, -1), w, pre + "o")


def latent_attention(h, w, pre, m, eps, places, cache):
    """Every head's keys and values are made anew from the cached latents."""
    T, H, rank = len(h), m["heads"], m["kv_rank"]
    q = linear(h, w, pre + "q").reshape(T, H, m["dim"] + m["rot_dim"])
    down = linear(h, w, pre + "dkv")
    c, part = rms(down[:, :rank], w[pre + "dkv.norm"], eps), rotate(down[:, None, rank:], places, m["rot"])[:, 0]
    q = np.concatenate([q[..., :m["dim"]], rotate(q[..., m["dim"]:], places, m["rot"])], -1)
    c, part = keep(cache, latents=c, parts=part)
    k = (c @ f64(w[pre + "uk"]).T).reshape(len(c), H, m["dim"])
    k = np.concatenate([k, np.broadcast_to(part[:, None], (len(c), H, m["rot_dim"]))], -1)
    v = (c @ f64(w[pre + "uv"]).T).reshape(len(c), H, m["vdim"])
    return linear(attend(q, k, v, places, m["scale"], m["mask"]["size"]).reshape(T, -1), w, pre + "o")


# ---- feed-forward

def dense(h, w, pre, m):
    return linear(gelu(linear(h, w, pre + "gate")) * linear(h, w, pre + "up"), w, pre + "down")


def expert(h, w, pre, limit):
    g, u = np.minimum(linear(h, w, pre + "gate"), limit), np.clip(linear(h, w, pre + "up"), -limit, limit)
    return linear(g * sigmoid(SLOPE * g) * (u + 1), w, pre + "down")


def route(h, w, pre, r):
    """(chosen experts, their weights) of each token: chosen by corrected scores, weighted by the scores themselves."""
    z = linear(h, w, pre + "router")
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    picks = np.argsort(-(s + w[pre + "correction"]), axis=-1, kind="stable")[:, :r["top"]]
    mine = np.take_along_axis(s, picks, -1)
    return picks, mine / (mine.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def mixture(h, w, pre, m):
    """The experts past the last real one give back their input."""
    picks, weight = route(h, w, pre, m["router"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(picks[t], weight[t]):
            out[t] += s * (expert(h[t:t + 1], w, f"{pre}e{e}.", m["expert"]["limit"])[0] if e < m["router"]["experts"] else h[t])
    return out


MIXERS = {"attention": attention, "attention_2": attention_2, "latent_attention": latent_attention}


def layer(x, w, i, entry, eps, places, cache):
    pre = f"l{i}."
    x = x + MIXERS[entry["type"]](rms(x, w[pre + "norm1"], eps), w, pre + "mix.", entry["mixer"], eps, places, cache)
    if entry.get("mlp"):
        h = rms(x, w[pre + "norm2"], eps)
        x = x + (dense if entry["mlp"]["kind"] == "dense" else mixture)(h, w, pre + "mlp.", entry["mlp"])
    return x


def order(cfg):
    """The layer runs in order: (layer, number of the pass that begins with it, or None)."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    once = range(start, stop)
    return [(i, None) for i in range(start)] + [(i, t if i == start else None) for t in range(loop["times"]) for i in once] + [(i, None) for i in range(stop, n)]


def pass_start(x, x0, w, t):
    return np.concatenate([x, x0], -1) @ f64(w["loop.in"]).T + w["loop.step"][t]


def embed(ids, w, cfg):
    return f64(w["embed"])[list(ids)] * cfg["embedding"]["scale"]


def head(x, w, cfg):
    return rms(x, w["final.norm"], cfg["norm"]["eps"]) @ f64(w["embed"]).T * cfg["logit_scale"]


def forward(ids, first, w, cfg, caches, residuals=None):
    """Logits of every token of ids, at places first.., one sequence; caches: a dict a layer run (start with empty ones).
    residuals: a list that receives the residual stream after every layer run."""
    places = list(range(first, first + len(ids)))
    x = x0 = embed(ids, w, cfg)
    for (i, t), cache in zip(order(cfg), caches):
        if t is not None:
            x = pass_start(x, x0, w, t)
        x = layer(x, w, i, cfg["layers"][i], cfg["norm"]["eps"], places, cache)
        if residuals is not None:
            residuals.append(x)
    return head(x, w, cfg)


def caches(cfg):
    return [{} for _ in order(cfg)]


def tensors(cfg):
    """{name: shape} of a configuration's checkpoint."""
    d = cfg["width"]
    out = {"embed": [cfg["vocab"], d]}
    if cfg.get("loop"):
        out |= {"loop.in": [d, 2 * d], "loop.step": [cfg["loop"]["times"], d]}
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        x, H = p + "mix.", m["heads"]
        out[p + "norm1"] = [d]
        if e["type"] == "latent_attention":
            out |= {x + "q": [H * (m["dim"] + m["rot_dim"]), d], x + "dkv": [m["kv_rank"] + m["rot_dim"], d], x + "dkv.norm": [m["kv_rank"]],
                    x + "uk": [H * m["dim"], m["kv_rank"]], x + "uv": [H * m["vdim"], m["kv_rank"]], x + "o": [d, H * m["vdim"]]}
        elif e["type"] == "attention":
            for name, n in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                out |= {x + name: [n, d], f"{x}{name}.conv": [n, m["conv"]]}
            out[x + "o"] = [d, H * m["vdim"]]
        else:
            for name, n in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"])):
                out |= {x + name: [n, d], f"{x}{name}.b": [n], f"{x}{name}.norm": [n]}
            out |= {x + "o": [d, H * m["vdim"]], x + "o.b": [d]}
        f = e.get("mlp")
        if not f:
            continue
        out[p + "norm2"] = [d]
        unit = lambda pre, ff, b: {pre + n + s: shape[:1] if s else shape for n, shape in (("gate", [ff, d]), ("up", [ff, d]), ("down", [d, ff])) for s in ([""] + [".b"] * b)}
        if f["kind"] == "dense":
            out |= unit(p + "mlp.", f["ff"], True)
        else:
            for j in range(f["router"]["experts"]):
                out |= unit(f"{p}mlp.e{j}.", f["expert"]["ff"], False)
            n = f["router"]["experts"] + f["router"]["identity"]
            out |= {p + "mlp.router": [n, d], p + "mlp.correction": [n]}
    out["final.norm"] = [d]
    return out
