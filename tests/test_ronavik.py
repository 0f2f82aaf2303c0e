"""Ronavik on the host: its configuration and checkpoint as the loader reads them, the oracle against itself however a sequence is
cut, mistakes planted in the oracle (each must show), the slot engine over a backend played by the oracle."""
import copy
from types import SimpleNamespace as NS

import numpy as np
import pytest

import ronavik_models as models
from oracle import ronavik as oracle


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
def test_a_checkpoint_loads_by_its_config(tmp_path, name):
    from ferrite_b200 import checkpoint, models as registry, ronavik
    cfg = models.CONFIGS[name]
    raw = models.weights(cfg)
    c, w = checkpoint.load(models.save(tmp_path, cfg, raw), places=77)
    assert registry.of(c) is ronavik
    assert (c.family, c.dim, c.vocab, c.layers, c.places, c.positions, c.eps) == ("ronavik", cfg["width"], cfg["vocab"], len(cfg["layers"]), 77, cfg["max_positions"], cfg["norm"]["eps"])
    exact, served = ronavik.precision(c, "fp32"), ronavik.precision(c, "bfp8")
    for i, e in enumerate(cfg["layers"]):
        p, x, m = f"l{i}.", f"l{i}.mix.", e["mixer"]
        if e["type"] == "parallel":
            own = [raw[x + n] for n in ("left.q", "left.k", "left.v", "right.y", "right.x")]
            assert np.array_equal(w[x + "o"].values().T, np.concatenate([raw[x + "left.o"], raw[x + "right.o"]], 1))
            part = m["right"]["width"] // m["right"]["blocks"]
            gates = w[x + "gates"].values()
            assert gates.shape == (m["right"]["blocks"], part, 2 * part) and np.array_equal(gates[-1].T, np.concatenate([raw[x + "right.ra"][-1], raw[x + "right.ri"][-1]]))
            assert np.array_equal(w[x + "gates.b"].values(), np.concatenate([raw[x + "right.ra.b"], raw[x + "right.ri.b"]], 1))
            assert np.array_equal(w[x + "conv"].values(), raw[x + "right.conv"].T) and np.array_equal(w[x + "lam"].values()[0], raw[x + "right.lam"]) and np.array_equal(w[x + "pb"].values()[0], raw[x + "left.pb"])
        else:
            own = [raw[x + "in"]]
            assert np.array_equal(w[x + "conv"].values(), raw[x + "conv"].T) and np.array_equal(w[x + "A_log"].values()[0], raw[x + "A_log"])
        assert np.array_equal(w[p + "in"].values().T, np.concatenate([raw[p + "rg1"]] + own))
        shapes = ronavik.projections(c, i)
        assert w[p + "in"].values().shape == shapes["in"] and w[x + "o"].values().shape == shapes["mix.o"]
        if e["mlp"]:
            n = e["mlp"]["router"]["experts"]
            assert np.array_equal(w[p + "mlp.in"].values().T, np.concatenate([raw[p + "rg2"], raw[p + "mlp.router"]])) and w[p + "mlp.in"].values().shape == shapes["mlp.in"]
            assert np.array_equal(w[p + "mlp.up"].values()[n - 1].T, raw[f"{p}mlp.e{n - 1}.up"]) and np.array_equal(w[p + "mlp.down"].values()[0].T, raw[p + "mlp.e0.down"])
        for op, (k, n) in shapes.items():
            assert ronavik.weight_format(p + op, exact) == "fp32" and ronavik.weight_format(p + op, served) == ("bf16" if op.startswith("mlp.") or n % 16 or k % 4 else "bfp8")
    assert ronavik.weight_format("l0.norm1b", served) == "fp32" and ronavik.weight_format("pos", served) == ronavik.weight_format("l0.mix.gates", served) == "bf16"
    assert not [n for n in w if ".e0." in n or ".left." in n or ".right." in n or ".rg1" == n[-4:] or n.endswith(".rg2")]


def test_what_a_layer_keeps():
    from ferrite_b200 import ronavik
    made = []
    c = ronavik.config(models.CONFIGS["mixed"])
    kv = ronavik.kv_cache(c, 60, lambda shape, dtype: made.append((shape, dtype)) or NS(), 3)
    assert len(kv) == 5 and [x[0] is None for x in kv] == [True, False, False, True, True]
    assert made[:2] == [((3, 3, 6 * 24 + 2 * 2 * 32), "fp32"), ((3, 6 * 32, 24), "fp32")]
    assert made[2:5] == [((2, 60, 32 + 40), "bf16"), ((3, 2, 64), "fp32"), ((3, 1, 64), "fp32")]


@pytest.mark.parametrize("change,what", [(lambda c: c["layers"][3].update(type="stroll"), "stroll"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse"), (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "whole groups of query"),
                                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "9 of 6"), (lambda c: c["layers"][1]["mixer"]["right"].update(blocks=7), "equal blocks"),
                                         (lambda c: c["layers"][0]["mixer"].update(groups=4), "whole groups of heads"), (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "equal parts")])
def test_what_is_not_served_is_refused_by_name(change, what):
    from ferrite_b200 import ronavik
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    change(cfg)
    with pytest.raises(AssertionError, match=what):
        ronavik.config(cfg)


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
def test_the_oracle_does_not_depend_on_how_a_sequence_is_cut(name):
    cfg = models.CONFIGS[name]
    w = models.weights(cfg)
    ids = np.random.default_rng(1).integers(0, cfg["vocab"], 23).tolist()
    whole = models.Alone(cfg, w)(ids)
    for cuts in ([1] * 23, [2, 9, 12], [22, 1]):
        run, at, rows = models.Alone(cfg, w), 0, []
        for n in cuts:
            rows.append(run(ids[at:at + n]))
            at += n
        np.testing.assert_allclose(np.concatenate(rows), whole, rtol=1e-9, atol=1e-9)


def planted(what, cfg, w, patch):
    """cfg, w or the oracle itself changed by one mistake."""
    keep = NS(**{n: getattr(oracle, n) for n in ("temperature", "weigh", "attend", "short_convolution", "gate", "recurrence", "state_space", "rms", "silu", "gelu", "route", "expert", "gated", "embed", "linear", "layer")})
    replace = lambda name, f: patch.setattr(oracle, name, f)
    mixers = [e["mixer"] for e in cfg["layers"]]
    if what == "no temperature":
        replace("temperature", lambda p, t: 1.0)
    elif what == "temperature from the place before":
        replace("temperature", lambda p, t: keep.temperature(max(p - 1, 0), t))
    elif what == "temperature without a floor":
        replace("temperature", lambda p, t: 1 + t["coef"] * np.log((p + 1) / t["every"] + 1))
    elif what == "softmax":
        replace("weigh", lambda s, b: np.exp(s - s.max()) / np.exp(s - s.max()).sum())
    elif what == "weights over their sum":
        replace("weigh", lambda s, b: keep.weigh(s, b) / keep.weigh(s, b).sum())
    elif what == "scaled after the bias":
        replace("attend", lambda q, k, v, places, scale, bias: keep.attend(q, k, v, places, scale, f64(bias) * scale))
    elif what == "one key more":
        replace("attend", lambda q, k, v, places, scale, bias: keep.attend(q, k, v, [min(p + 1, len(k) - 1) for p in places], scale, bias))
    elif what == "the first key unseen":
        replace("attend", lambda q, k, v, places, scale, bias: keep.attend(q, k, np.concatenate([0 * v[:1], v[1:]]), places, scale, bias))
    elif what == "key heads in turn":
        replace("attend", lambda q, k, v, places, scale, bias: keep.attend(q, k[:, np.arange(q.shape[1]) % k.shape[1]], v[:, np.arange(q.shape[1]) % k.shape[1]], places, scale, bias))
    elif what == "scale":
        mixers[1]["left"]["scale"] *= 1.02
    elif what in ("left scale", "right scale"):
        mixers[1][what.replace(" ", "_")] *= 1.02
    elif what == "taps reversed":
        replace("short_convolution", lambda u, v, name, cache: keep.short_convolution(u, v | {name: v[name][:, ::-1]}, name, cache))
    elif what in ("a lost convolution state", "a lost state"):
        name = "conv" if "conv" in what else "state"
        replace("layer", lambda x, v, i, e, eps, places, cache: [cache.pop(n) for n in list(cache) if n.endswith(name)] and None or keep.layer(x, v, i, e, eps, places, cache))
    elif what == "SiLU on the recurrence's input":
        replace("short_convolution", lambda u, v, name, cache: (lambda y: keep.silu(y) if ".right." in name else y)(keep.short_convolution(u, v, name, cache)))
    elif what == "gates exchanged":
        replace("recurrence", lambda u, r, i, lam, s: keep.recurrence(u, i, r, lam, s))
    elif what == "gates' matrices turned":
        replace("gate", lambda u, v, name: keep.gate(u, v | {name: np.swapaxes(v[name], 1, 2)}, name))
    elif what == "one gate for all blocks":
        replace("gate", lambda u, v, name: keep.gate(u, v | {name: v[name][:1].repeat(len(v[name]), 0)}, name))
    elif what == "a plain sum":  # without sqrt(1 - a^2)
        def recurrence(u, r, i, lam, s):
            out = np.zeros_like(u)
            for t in range(len(u)):
                s = np.exp(-8 * r[t] * oracle.softplus(lam)) * s + i[t] * u[t]
                out[t] = s
            return out, s
        replace("recurrence", recurrence)
    elif what == "a first token of its own":  # the whole of it enters the state
        def recurrence(u, r, i, lam, s):
            out, last = keep.recurrence(u, r, i, lam, s)
            if not np.any(s):
                first = np.exp(-8 * r[0] * oracle.softplus(f64(lam)))
                out, last = keep.recurrence(np.concatenate([u[:1] / np.sqrt(1 - first ** 2), u[1:]]), r, i, lam, s)
            return out, last
        replace("recurrence", recurrence)
    elif what == "another rate":
        replace("recurrence", lambda u, r, i, lam, s: keep.recurrence(u, r * 1.02, i, lam, s))
    elif what == "erf":  # GELU's other form
        from math import erf
        replace("gelu", lambda z: 0.5 * z * (1 + np.vectorize(erf)(z / np.sqrt(2))))
    elif what == "groups in turn":
        def state_space(x, b, c, dt, a, s):
            h = np.arange(x.shape[1]) % b.shape[1]
            return keep.state_space(x, b[:, h], c[:, h], dt, a, s)
        replace("state_space", state_space)
    elif what == "keys and queries exchanged":
        replace("state_space", lambda x, b, c, dt, a, s: keep.state_space(x, c, b, dt, a, s))
    elif what == "a step of one":
        replace("state_space", lambda x, b, c, dt, a, s: keep.state_space(x / dt[..., None], b, c, dt, a, s))
    elif what == "the gate after the norm":
        def mamba2(h, v, pre, m, eps, places, cache):
            z = keep.linear(h, v, pre + "in")[:, :m["heads"] * m["vdim"]]
            seen = {}
            replace("rms", lambda x, n, e: seen.setdefault("y", keep.rms(x / keep.silu(z).reshape(x.shape), n, e) * keep.silu(z).reshape(x.shape)) if x.ndim == 3 else keep.rms(x, n, e))
            out = oracle.mamba2(h, v, pre, m, eps, places, cache)
            replace("rms", keep.rms)
            return out
        patch.setitem(oracle.MIXERS, "mamba2", mamba2)
    elif what == "one norm for all parts":
        for m in mixers:
            if "norm_groups" in m:
                m["norm_groups"] = 1
    elif what == "weights on the output":
        def mixture(h, v, pre, m):
            out = np.zeros_like(h)
            for t, (picks, weights) in enumerate(zip(*keep.route(h, v, pre, m["router"]))):
                for e, s in zip(picks, weights):
                    out[t] += s * keep.expert(h[t:t + 1], v, f"{pre}e{e}.")[0]
            return out
        replace("mixture", mixture)
    elif what == "softmax scores":
        def route(h, v, pre, r):
            z = keep.linear(h, v, pre + "router")
            e = np.exp(z - z.max(-1, keepdims=True))
            picks, _ = keep.route(h, v, pre, r)
            return picks, np.take_along_axis(e / e.sum(-1, keepdims=True), picks, -1)
        replace("route", route)
    elif what == "one expert less":
        cfg["layers"][1]["mlp"]["router"]["top"] -= 1
    elif what == "plain ReLU":
        replace("expert", lambda h, v, pre: keep.linear(np.maximum(keep.linear(h, v, pre + "up"), 0), v, pre + "down"))
    elif what == "the gate of the result reads the result":
        replace("gated", lambda y, h, v, name: keep.gated(y, y, v, name))
    elif what in ("no gate rg1", "no gate rg2"):
        replace("gated", lambda y, h, v, name: y if name.endswith(what[-3:]) else keep.gated(y, h, v, name))
    elif what == "the gate after the norm of the result":
        held = {}
        def gated(y, h, v, name):
            held["gate"] = oracle.sigmoid(keep.linear(h, v, name))
            return y
        def rms(x, v, eps):
            g = held.pop("gate", None)
            return keep.rms(x, v, eps) * (1 if g is None else g)
        replace("gated", gated), replace("rms", rms)
    elif what == "places from 1":
        replace("embed", lambda ids, places, v: keep.embed(ids, [p + 1 for p in places], v))
    elif what == "eps":
        cfg["norm"]["eps"] = 1e-3
    else:  # a tensor left out
        assert what in w, what
        w[what] = np.ones_like(w[what]) if what.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")) else np.zeros_like(w[what])


f64 = np.float64
MISTAKES = ["no temperature", "temperature from the place before", "temperature without a floor", "softmax", "weights over their sum", "scaled after the bias", "one key more", "the first key unseen", "key heads in turn", "scale",
            "left scale", "right scale", "taps reversed", "a lost convolution state", "a lost state", "SiLU on the recurrence's input", "gates exchanged", "gates' matrices turned", "one gate for all blocks", "a plain sum",
            "a first token of its own", "another rate", "groups in turn", "keys and queries exchanged", "a step of one", "the gate after the norm", "one norm for all parts", "weights on the output",
            "softmax scores", "one expert less", "plain ReLU", "the gate of the result reads the result", "no gate rg1", "no gate rg2", "the gate after the norm of the result", "places from 1", "eps"]
TENSORS = ["pos", "l0.norm1", "l0.norm1b", "l0.norm2", "l1.norm2b", "final.norm", "l0.rg1.b", "l1.rg2.b", "l0.mix.conv.b", "l0.mix.dt_bias", "l0.mix.A_log", "l0.mix.D", "l0.mix.norm", "l1.mix.left.q.norm", "l1.mix.left.k.norm",
           "l1.mix.left.pb", "l1.mix.right.y.b", "l1.mix.right.x.b", "l1.mix.right.conv.b", "l1.mix.right.ra.b", "l1.mix.right.ri.b", "l1.mix.right.lam"]


@pytest.mark.parametrize("what", MISTAKES + TENSORS)
def test_the_weights_show_a_mistake(what, monkeypatch):
    # each is far above what the tests allow the device in fp32
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    w = models.weights(cfg)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 60).tolist()

    def run():
        one = models.Alone(cfg, w)
        return np.concatenate([one(ids[:40]), one(ids[40:42]), one(ids[42:])])
    want = run()
    planted(what, cfg, w, monkeypatch)
    assert models.error(run(), want) > 0.002


def test_no_choice_of_experts_is_a_close_call():
    for name, cfg in models.CONFIGS.items():
        w = models.weights(cfg)
        ids = np.random.default_rng(4).integers(0, cfg["vocab"], 40).tolist()
        seen = []
        keep, oracle.route = oracle.route, lambda h, v, pre, r: seen.append((oracle.linear(h, v, pre + "router"), np.abs(h).max(), r["top"])) or keep(h, v, pre, r)
        try:
            models.Alone(cfg, w)(ids)
        finally:
            oracle.route = keep
        assert seen
        for z, most, top in seen:
            if top < z.shape[1]:
                s = np.sort(z, -1)[:, ::-1]
                assert (s[:, top - 1] - s[:, top]).min() > 0.02, name  # (a logit's rounding in bf16 is less than a tenth of that)


class OracleBackend:
    """The engine's device side played by the oracle."""
    rewinds = False

    def __init__(self, cfg, w, slots):
        self.cfg, self.w, self.caches = cfg, w, [oracle.caches(cfg) for _ in range(slots)]

    def run(self, u, ids, first):
        if first == 0:
            self.caches[u] = oracle.caches(self.cfg)
        logits = oracle.forward(ids, first, self.w, self.cfg, self.caches[u])[-1]
        order = np.argsort(-logits, kind="stable")[:64]
        return logits[order], order, 0.0

    def prefill(self, u, ids, first, t):
        return self.run(u, ids, first)

    def decode(self, ids, places, ts):
        return [self.run(u, [i], p) if p < 63 else None for u, (i, p) in enumerate(zip(ids, places))]


def test_engine_reuses_a_slot_whole_or_not_at_all():
    from ferrite_b200 import ronavik
    from ferrite_b200.serve import Engine, Request
    assert ronavik.REWINDS is False
    cfg = models.CONFIGS["mixed"]
    w = models.weights(cfg)
    rng = np.random.default_rng(3)
    draw = lambda n: rng.integers(0, cfg["vocab"], n).tolist()
    engine = Engine(OracleBackend(cfg, w, 2), slots=2, places=64, chunk=4)
    first = engine.run([Request(draw(9), max_tokens=5)])[0]
    held = first.ids + first.made[:-1]
    rs = engine.run([Request(held + [3, 4], max_tokens=4), Request(first.ids[:5] + [7], max_tokens=6), Request(draw(2), max_tokens=3)])
    assert [r.cached for r in rs] == [len(held), 0, 0]
    assert all(r.made == models.greedy(cfg, w, r.ids, r.max_tokens) for r in [first] + rs)
