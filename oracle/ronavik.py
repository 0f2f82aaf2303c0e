"""TEST INFRASTRUCTURE (not the product): the Ronavik decoder as plain numpy in float64, one function per mechanism, token by
token, query by query and expert by expert.  Weights are {name: array} under the checkpoint's own tensor names (linear weights
[out, in]); the configuration is the parsed config.json."""
import math

import numpy as np


def f64(x):
    return np.asarray(x, np.float64)


def sigmoid(x):
    return 1 / (1 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0, x)


def gelu(z):
    return 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def linear(h, w, name):
    """W h, and the bias where the checkpoint has one."""
    y = h @ f64(w[name]).T
    return y + w[name + ".b"] if name + ".b" in w else y


def short_convolution(u, w, name, cache):
    """y_t = bias + sum_j kernel[:, j] u_(t - taps + 1 + j), a kernel a channel; u before the first token is 0.  The cache keeps
    the last taps - 1 rows of u."""
    kernel = f64(w[name])
    back = kernel.shape[1] - 1
    rows = np.concatenate([cache.get(name, np.zeros((back, u.shape[1]))), u])
    cache[name] = rows[len(rows) - back:]
    return sum(kernel[:, j] * rows[j:j + len(u)] for j in range(back + 1)) + w[name + ".b"]


# ---- attention whose weights are sigmoids

def temperature(place, t):
    """What a query at `place` is multiplied by."""
    return 1 + t["coef"] * math.log(math.floor((place + 1) / t["every"]) + 1)


def weigh(scores, bias):
    """A key's weight, from its own score alone."""
    return sigmoid(scores + bias)


def attend(q, k, v, places, scale, bias):
    """q [T, H, D] at places over k [L, G, D], v [L, G, V] of the places 0..L-1; a key head serves H / G query heads in a row."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t, p in enumerate(places):
        for h in range(H):
            out[t, h] = weigh(k[:p + 1, h // rep] @ q[t, h] * scale, bias[h]) @ v[:p + 1, h // rep]
    return out


def attention(h, w, pre, m, eps, places, cache):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q = rms(linear(h, w, pre + "q").reshape(T, H, m["dim"]), w[pre + "q.norm"], eps)
    q = q * np.array([temperature(p, m["q_temp"]) for p in places])[:, None, None]
    k = rms(linear(h, w, pre + "k").reshape(T, G, m["dim"]), w[pre + "k.norm"], eps)
    for name, x in (("keys", k), ("values", linear(h, w, pre + "v").reshape(T, G, m["vdim"]))):
        cache[name] = np.concatenate([cache[name], x]) if name in cache else x
    return linear(attend(q, cache["keys"], cache["values"], places, m["scale"], w[pre + "pb"]).reshape(T, -1), w, pre + "o")


# ---- a gated linear recurrence

def gate(u, w, name):
    """A sigmoid of each part of u by a matrix of its own."""
    blocks = len(w[name])
    parts = u.reshape(len(u), blocks, -1)
    return sigmoid(np.concatenate([parts[:, b] @ f64(w[name][b]).T + w[name + ".b"][b] for b in range(blocks)], -1))


def recurrence(u, r, i, lam, state):
    """S = a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); every token's S."""
    out = np.zeros_like(u)
    for t in range(len(u)):
        a = np.exp(-8 * r[t] * softplus(f64(lam)))
        state = a * state + np.sqrt(1 - a * a) * i[t] * u[t]
        out[t] = state
    return out, state


def recurrent_block(h, w, pre, m, cache):
    y = gelu(linear(h, w, pre + "y"))
    u = short_convolution(linear(h, w, pre + "x"), w, pre + "conv", cache)
    s, cache["state"] = recurrence(u, gate(u, w, pre + "ra"), gate(u, w, pre + "ri"), w[pre + "lam"], cache.get("state", np.zeros(u.shape[1])))
    return linear(s * y, w, pre + "o")


def parallel(h, w, pre, m, eps, places, cache):
    left, right = attention(h, w, pre + "left.", m["left"], eps, places, cache), recurrent_block(h, w, pre + "right.", m["right"], cache)
    return m["left_scale"] * left + m["right_scale"] * right


# ---- a state space with a decay per token and head

def state_space(x, b, c, dt, a_log, state):
    """S_h = exp(-exp(a_log) dt) S_h + dt b x^T, y = S_h^T c; x [T, H, P], b and c [T, G, N], dt [T, H], state [H, N, P]."""
    T, H = x.shape[:2]
    rep, state, out = H // b.shape[1], state.copy(), np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            state[h] = np.exp(-np.exp(f64(a_log[h])) * dt[t, h]) * state[h] + dt[t, h] * np.outer(b[t, h // rep], x[t, h])
            out[t, h] = state[h].T @ c[t, h // rep]
    return out, state


def mamba2(h, w, pre, m, eps, places, cache):
    T, H, P, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = np.split(linear(h, w, pre + "in"), [inner, 2 * inner + 2 * G * N], axis=-1)
    x, b, c = np.split(silu(short_convolution(xbc, w, pre + "conv", cache)), [inner, inner + G * N], axis=-1)
    x = x.reshape(T, H, P)
    y, cache["state"] = state_space(x, b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], cache.get("state", np.zeros((H, N, P))))
    y = ((y + f64(w[pre + "D"])[:, None] * x).reshape(T, inner) * silu(z)).reshape(T, m["norm_groups"], -1)
    return linear(rms(y, 1.0, eps).reshape(T, inner) * w[pre + "norm"], w, pre + "o")


# ---- feed-forward

def expert(h, w, pre):
    return linear(np.maximum(linear(h, w, pre + "up"), 0) ** 2, w, pre + "down")


def route(h, w, pre, r):
    """(chosen experts, their weights) of each token: each output's own sigmoid both chooses and weighs."""
    z = linear(h, w, pre + "router")
    picks = np.argsort(-z, axis=-1, kind="stable")[:, :r["top"]]
    return picks, sigmoid(np.take_along_axis(z, picks, -1))


def mixture(h, w, pre, m):
    """An expert's weight is on its input."""
    out = np.zeros_like(h)
    for t, (picks, weights) in enumerate(zip(*route(h, w, pre, m["router"]))):
        for e, s in zip(picks, weights):
            out[t] += expert(s * h[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


# ---- the decoder

MIXERS = {"parallel": parallel, "mamba2": mamba2}


def gated(y, h, w, name):
    """A sublayer's result times a sigmoid of what the sublayer read."""
    return y * sigmoid(linear(h, w, name))


def layer(x, w, i, entry, eps, places, cache):
    pre = f"l{i}."
    h = rms(x, w[pre + "norm1"], eps)
    x = x + rms(gated(MIXERS[entry["type"]](h, w, pre + "mix.", entry["mixer"], eps, places, cache), h, w, pre + "rg1"), w[pre + "norm1b"], eps)
    if entry.get("mlp"):
        h = rms(x, w[pre + "norm2"], eps)
        x = x + rms(gated(mixture(h, w, pre + "mlp.", entry["mlp"]), h, w, pre + "rg2"), w[pre + "norm2b"], eps)
    return x


def embed(ids, places, w):
    return f64(w["embed"])[list(ids)] + f64(w["pos"])[list(places)]


def head(x, w, eps):
    return rms(x, w["final.norm"], eps) @ f64(w["embed"]).T


def forward(ids, first, w, cfg, caches, residuals=None):
    """Logits of every token of ids, at places first.., one sequence; caches: a dict a layer (start with empty ones).
    residuals: a list that receives the residual stream after every layer."""
    places, eps = list(range(first, first + len(ids))), cfg["norm"]["eps"]
    x = embed(ids, places, w)
    for i, (entry, cache) in enumerate(zip(cfg["layers"], caches)):
        x = layer(x, w, i, entry, eps, places, cache)
        if residuals is not None:
            residuals.append(x)
    return head(x, w, eps)


def caches(cfg):
    return [{} for _ in cfg["layers"]]


def tensors(cfg):
    """{name: shape} of a configuration's checkpoint."""
    d = cfg["width"]
    out = {"embed": [cfg["vocab"], d], "pos": [cfg["max_positions"], d]}
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        x = p + "mix."
        out |= {p + "norm1": [d], p + "norm1b": [d], p + "rg1": [d, d], p + "rg1.b": [d]}
        if e["type"] == "mamba2":
            inner, joint = m["heads"] * m["vdim"], m["groups"] * m["state"] * 2
            out |= {x + "in": [2 * inner + joint + m["heads"], d], x + "conv": [inner + joint, m["conv"]], x + "conv.b": [inner + joint]}
            out |= {x + n: [m["heads"]] for n in ("dt_bias", "A_log", "D")} | {x + "norm": [inner], x + "o": [d, inner]}
        else:
            l, r, a, b = m["left"], m["right"], x + "left.", x + "right."
            out |= {a + "q": [l["heads"] * l["dim"], d], a + "k": [l["kv_heads"] * l["dim"], d], a + "v": [l["kv_heads"] * l["vdim"], d], a + "q.norm": [l["dim"]], a + "k.norm": [l["dim"]],
                    a + "pb": [l["heads"]], a + "o": [d, l["heads"] * l["vdim"]]}
            n, part = r["width"], [r["blocks"], r["width"] // r["blocks"]]
            out |= {b + "y": [n, d], b + "y.b": [n], b + "x": [n, d], b + "x.b": [n], b + "conv": [n, r["conv"]], b + "conv.b": [n], b + "lam": [n], b + "o": [d, n]}
            out |= {b + g + s: part + ([] if s else part[1:]) for g in ("ra", "ri") for s in ("", ".b")}
        f = e.get("mlp")
        if f:
            out |= {p + "norm2": [d], p + "norm2b": [d], p + "rg2": [d, d], p + "rg2.b": [d], p + "mlp.router": [f["router"]["experts"], d]}
            for j in range(f["router"]["experts"]):
                out |= {f"{p}mlp.e{j}.up": [f["expert"]["ff"], d], f"{p}mlp.e{j}.down": [d, f["expert"]["ff"]]}
    out["final.norm"] = [d]
    return out
