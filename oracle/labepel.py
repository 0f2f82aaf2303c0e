"""TEST INFRASTRUCTURE (not the product): the Labepel decoder as plain numpy in float64, one function per mechanism, key by
key and expert by expert.  Weights are {name: array} under the checkpoint's own tensor names (linear weights [out, in]); the
configuration is the parsed config.json."""
import math

import numpy as np

f64 = np.float64


def sigmoid(x):
    return 1 / (1 + np.exp(-x))


def rms(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def chunk_of(place, size):
    """The first place of the chunk a place lies in."""
    return place // size * size


def attend(q, k, v, places, size, scale):
    """q [T, H, D] at places; k [L, G, D], v [L, G, V] of the places 0..L-1: softmax over the keys of each query's chunk up to
    itself, a key group shared by H / G query heads in a row; one more term, exp(0), stands in the denominator."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t, p in enumerate(places):
        seen = slice(chunk_of(p, size), p + 1)
        for h in range(H):
            g = h // (H // G)
            s = k[seen, g] @ q[t, h] * scale
            m = max(s.max(), 0.0)
            e = np.exp(s - m)
            out[t, h] = e @ v[seen, g] / (e.sum() + math.exp(-m))
    return out


def project(h, w, name):
    return h @ w[name].T + w[name + ".b"]


def mix_values(v, first, share):
    """The layer's values and the first mixing layer's of the same token; the first such layer's are its own."""
    return v if first is None else (1 - share) * v + share * first.reshape(v.shape)


def attention(h, w, pre, m, eps, places, cache, shared):
    """cache: what this layer keeps of the sequence (keys and values by place); shared: the forward pass's, with the first
    mixing layer's values."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms(project(h, w, pre + "q").reshape(T, H, m["dim"]), w[pre + "q.norm"], eps)
    k = rms(project(h, w, pre + "k").reshape(T, G, m["dim"]), w[pre + "k.norm"], eps)
    v = project(h, w, pre + "v").reshape(T, G, m["vdim"])
    if m.get("v_mix"):
        first = shared.setdefault("v", None)
        shared["v"] = v if first is None else first
        v = mix_values(v, first, f64(w[pre + "vmix"].reshape(())) if first is not None else 0.0)
    for name, x in (("k", k), ("v", v)):
        cache[name] = np.concatenate([cache[name], x]) if name in cache else x
    o = attend(q, cache["k"], cache["v"], places, m["mask"]["size"], m["scale"]).reshape(T, H * m["vdim"])
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def gated(h, w, pre):
    g = h @ w[pre + "gate"].T
    return (g * sigmoid(g) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(h, w, pre, m):
    """(chosen experts, their weights) of each token."""
    z = h @ w[pre + "router"].T + w[pre + "router.b"]
    picks = np.argsort(-z, axis=-1, kind="stable")[:, :m["router"]["top"]]
    e = np.take_along_axis(z, picks, -1)
    e = np.exp(e - e.max(-1, keepdims=True))
    return picks, e / e.sum(-1, keepdims=True)


def mixture(h, w, pre, m, picks=None):
    """picks: another run's choices (each token's own weights still follow from its logits)."""
    chosen, weight = route(h, w, pre, m)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], weight[t]):
            out[t] += s * gated(h[t:t + 1], w, f"{pre}e{e}.")[0]
    return out + gated(h, w, pre + "shared.") if m.get("shared") else out


def layer(x, w, i, entry, eps, places, cache, shared):
    """Mixer and feed-forward read the same normed rows; each result is scaled by column and both are added."""
    pre = f"l{i}."
    h = rms(x, 1 + f64(w[pre + "norm1"]), eps)
    y = attention(h, w, pre + "mix.", entry["mixer"], eps, places, cache, shared) * w[pre + "ls1"]
    if entry.get("mlp"):
        y = y + mixture(h, w, pre + "mlp.", entry["mlp"]) * w[pre + "ls2"]
    return x + y


def forward(ids, first, w, cfg, caches, residuals=None):
    """Logits of every token of ids, at places first.., one sequence; caches: a list of dicts, one a layer (start with
    empty ones).  residuals: a list that receives the residual stream after every layer."""
    places = list(range(first, first + len(ids)))
    x = f64(w["embed"])[list(ids)] + f64(w["pos"])[places]
    shared = {}
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, w, i, entry, cfg["norm"]["eps"], places, caches[i], shared)
        if residuals is not None:
            residuals.append(x)
    return rms(x, 1 + f64(w["final.norm"]), cfg["norm"]["eps"]) @ f64(w["embed"]).T


def caches(cfg):
    return [{} for _ in cfg["layers"]]


def tensors(cfg):
    """{name: shape} of a configuration's checkpoint."""
    d = cfg["width"]
    out = {"embed": [cfg["vocab"], d], "pos": [cfg["max_positions"], d]}

    def unit(pre, ff):
        out.update({pre + "gate": [ff, d], pre + "up": [ff, d], pre + "down": [d, ff]})
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        H, G = m["heads"], m["kv_heads"]
        out[p + "norm1"] = [d]
        for name, n in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"])):
            out |= {f"{p}mix.{name}": [n, d], f"{p}mix.{name}.b": [n]}
        out |= {p + "mix.q.norm": [m["dim"]], p + "mix.k.norm": [m["dim"]], p + "mix.g": [H * m["vdim"], d], p + "mix.o": [d, H * m["vdim"]], p + "ls1": [d]}
        if m.get("v_mix"):
            out[p + "mix.vmix"] = []
        if e.get("mlp"):
            f = e["mlp"]
            for j in range(f["router"]["experts"]):
                unit(f"{p}mlp.e{j}.", f["expert"]["ff"])
            out |= {p + "mlp.router": [f["router"]["experts"], d], p + "mlp.router.b": [f["router"]["experts"]], p + "ls2": [d]}
            if f.get("shared"):
                unit(p + "mlp.shared.", f["shared"]["ff"])
    out["final.norm"] = [d]
    return out
