"""Vunadra on the host: its configuration and checkpoint as the loader reads them, frequencies, the oracle against itself however a
sequence is cut, mistakes planted in the oracle (each must show), the slot engine over a backend played by the oracle."""
import copy
from types import SimpleNamespace as NS

import numpy as np
import pytest

import vunadra_models as models
from oracle import vunadra as oracle


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
def test_a_checkpoint_loads_by_its_config(tmp_path, name):
    from ferrite_b200 import checkpoint, models as registry, vunadra
    cfg = models.CONFIGS[name]
    raw = models.weights(cfg)
    c, w = checkpoint.load(models.save(tmp_path, cfg, raw), places=77)
    assert registry.of(c) is vunadra
    assert (c.family, c.dim, c.vocab, c.layers, c.places, c.eps) == ("vunadra", cfg["width"], cfg["vocab"], len(cfg["layers"]), 77, cfg["norm"]["eps"])
    assert (c.embed_scale, c.logit_scale, c.runs) == (cfg["embedding"]["scale"], cfg["logit_scale"], oracle.order(cfg))
    fmt, exact = vunadra.precision(c, "bf16"), vunadra.precision(c, "fp32")
    for i, e in enumerate(cfg["layers"]):
        m, p, j = c.blocks[i].mixer, f"l{i}.", e["mixer"]
        assert (m.heads, m.scale, m.window, m.rot.dims) == (j["heads"], j["scale"], j.get("mask", {}).get("size", 0), j["rot"]["dims"])
        names = dict(attention="qkv", attention_2="qk", latent_attention=("q", "dkv"))[e["type"]]
        assert np.array_equal(w[p + "mix.in"].values().T, np.concatenate([raw[p + "mix." + n] for n in names]))
        if e["type"] == "attention":
            assert np.array_equal(w[p + "mix.conv"].values(), np.concatenate([raw[f"{p}mix.{n}.conv"] for n in names]).T)
        elif e["type"] == "attention_2":
            assert np.array_equal(w[p + "mix.b"].values()[0], np.concatenate([raw[f"{p}mix.{n}.b"] for n in names])) and m.softcap == j["softcap"]
        else:
            assert np.array_equal(w[p + "mix.uk"].values().reshape(raw[p + "mix.uk"].shape), raw[p + "mix.uk"])
            assert np.array_equal(w[p + "mix.uv"].values()[-1].T, raw[p + "mix.uv"][-j["vdim"]:])
        assert (p + "mlp.gate_up" in w) == (p + "norm2" in w) == bool(e["mlp"])
        if e["mlp"] and e["mlp"]["kind"] == "moe":
            last = e["mlp"]["router"]["experts"] - 1
            assert w[p + "mlp.gate_up"].values().shape == (last + 1, cfg["width"], 2 * e["mlp"]["expert"]["ff"])
            assert np.array_equal(w[p + "mlp.down"].values()[last], raw[f"{p}mlp.e{last}.down"].T)
            assert np.array_equal(w[p + "mlp.router.b"].values()[0], raw[p + "mlp.correction"])
        for n in ("norm1", "norm2", "mix.b", "mix.conv", "mix.o.b", "mix.q.norm", "mix.dkv.norm", "mlp.gate_up.b", "mlp.down.b", "mlp.router.b"):
            assert vunadra.weight_format(p + n, fmt) == "fp32"
        for n in ("mix.in", "mix.uk", "mix.uv", "mix.o", "mlp.gate_up", "mlp.down", "mlp.router"):
            assert e["mlp"] is None and n.startswith("mlp") or (vunadra.weight_format(p + n, fmt), vunadra.weight_format(p + n, exact)) == ("bf16", "fp32")
    assert vunadra.weight_format("loop.in", fmt) == "bf16" and vunadra.weight_format("loop.step", fmt) == vunadra.weight_format("final.norm", fmt) == "fp32"
    assert vunadra.weight_format("head", exact) == vunadra.weight_format("embed", exact) == "fp32"


def test_block_float_formats_leave_experts_and_heads_matrices_alone():
    from ferrite_b200 import vunadra
    prec = vunadra.precision(vunadra.config(models.CONFIGS["mixed"]), "bfp8")
    of = lambda name: vunadra.weight_format(name, prec)
    assert of("l0.mix.in") == of("l0.mlp.gate_up") == of("l1.mix.o") == of("loop.in") == "bfp8"
    assert of("l1.mlp.gate_up") == of("l1.mlp.router") == of("l2.mix.uk") == of("l2.mix.uv") == "bf16"
    odd = vunadra.precision(vunadra.config(models.CONFIGS["odd"]), "bfp8")
    assert odd["mix.in", 0][0] == odd["loop.in", None][0] == "bf16", "no whole runs of 16 columns"


def test_a_loop_runs_its_layers_in_turn_with_caches_of_their_own():
    from ferrite_b200 import vunadra
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    cfg["loop"] = dict(start=1, stop=3, times=3)
    c = vunadra.config(cfg)
    assert c.runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]
    made = []
    kv = vunadra.kv_cache(c, 60, lambda shape, dtype: made.append((shape, dtype)) or NS(), 3)
    assert len(kv) == 9 and made.count(((1, 60, 48), "bf16")) == 3 and made.count(((2, 60, 32), "bf16")) == 4  # the latents' rows; the keys and values of attention_2
    assert ((3, 2, 6 * 24 + 2 * 40), "fp32") in made and ((3, 3, 6 * 24 + 2 * 40), "fp32") in made  # convolutions of 3 and 4 taps
    del cfg["loop"]
    assert vunadra.config(cfg | dict(loop=None)).runs == vunadra.config(cfg).runs == [(l, None) for l in range(5)]


@pytest.mark.parametrize("change,what", [(lambda c: c["layers"][3].update(type="stroll"), "stroll"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "whole groups"),
                                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "9 of 8"), (lambda c: c["layers"][1]["mixer"].update(vdim=8), "as wide"),
                                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "even number"), (lambda c: c["loop"].update(stop=6), "run of layers")])
def test_what_is_not_served_is_refused_by_name(change, what):
    from ferrite_b200 import vunadra
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    change(cfg)
    with pytest.raises(AssertionError, match=what):
        vunadra.config(cfg)


@pytest.mark.parametrize("rot", [dict(base=500.0, dims=24), dict(base=1e4, dims=64, scaling=dict(factor=4.0, original=512, fast=32.0, slow=1.0)), dict(base=50.0, dims=6, scaling=dict(factor=2.0, original=16, fast=2.0, slow=1.9)),
                                 dict(base=300.0, dims=16, scaling=dict(factor=3.0, high=4.0, low=1.0, original=96)), dict(base=5e5, dims=128, scaling=dict(factor=8.0, high=4.0, low=1.0, original=8192))])
def test_frequencies(rot):
    from ferrite_b200 import mixers
    f, mag = mixers.frequencies(NS(**rot | dict(scaling=NS(**rot["scaling"]) if "scaling" in rot else None)))
    want, want_mag = oracle.frequencies(rot)
    np.testing.assert_allclose(f, want, rtol=1e-12)
    assert mag == pytest.approx(want_mag, rel=1e-12)


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
    keep = {n: getattr(oracle, n) for n in ("attend", "route", "convolved", "rotate", "layer", "keep", "pass_start", "order", "expert", "frequencies", "rms", "attention_2")}
    mixers = [e["mixer"] for e in cfg["layers"]]
    if what in ("window 1 longer", "window 1 shorter", "window 2 longer", "window 2 shorter"):
        mixers[int(what.split()[1])]["mask"]["size"] += 1 if what.endswith("longer") else -1
    elif what == "no softcap":
        patch.setattr(oracle, "capped", lambda s, cap: s)
    elif what in ("scale 0", "scale 1", "scale 2"):
        mixers[int(what[-1])]["scale"] *= 1.03
    elif what == "turned halves":  # (i, i + dims / 2) in the place of neighbours
        def rotate(x, places, rot):
            n = rot["dims"]
            order = np.r_[np.arange(n).reshape(2, n // 2).T.reshape(-1), np.arange(n, x.shape[-1])]
            out = np.empty_like(x)
            out[..., order] = keep["rotate"](x[..., order], places, rot)
            return out
        patch.setattr(oracle, "rotate", rotate)
    elif what == "no magnitude":
        patch.setattr(oracle, "frequencies", lambda rot: (keep["frequencies"](rot)[0], 1.0))
    elif what in ("plain frequencies 0", "plain frequencies 1"):
        mixers[int(what[-1])]["rot"].pop("scaling")
    elif what == "places from 1":
        patch.setattr(oracle, "rotate", lambda x, places, rot: keep["rotate"](x, np.asarray(places) + (1 if x.shape[1] == 1 else 0), rot))
    elif what == "values after the norm":
        patch.setattr(oracle, "keep", lambda cache, **new: keep["keep"](cache, **new | (dict(values=new["keys"]) if "values" in new and new["values"].shape == new["keys"].shape else {})))
    elif what == "norm by head":
        patch.setattr(oracle, "rms", lambda x, v, eps: keep["rms"](x.reshape(len(x), 6, 16), v.reshape(6, 16), eps).reshape(x.shape) if x.shape[-1] == 96 and v is w["l1.mix.q.norm"] else keep["rms"](x, v, eps))
    elif what == "taps reversed":
        patch.setattr(oracle, "convolved", lambda u, kernel, before: keep["convolved"](u, kernel[:, ::-1], before))
    elif what == "a lost state":
        patch.setattr(oracle, "convolved", lambda u, kernel, before: keep["convolved"](u, kernel, np.zeros_like(before)))
    elif what == "weights with the correction":
        def route(h, w, pre, r):
            picks, _ = keep["route"](h, w, pre, r)
            z = oracle.linear(h, w, pre + "router")
            e = np.exp(z - z.max(-1, keepdims=True))
            s = np.take_along_axis(e / e.sum(-1, keepdims=True) + w[pre + "correction"], picks, -1)
            return picks, s / (s.sum(-1, keepdims=True) + 1e-20) * r["scale"]
        patch.setattr(oracle, "route", route)
    elif what == "choice without the correction":
        w["l1.mlp.correction"] = np.zeros_like(w["l1.mlp.correction"])
    elif what == "identity gives nothing":
        patch.setattr(oracle, "route", lambda h, v, pre, r: (lambda p, s: (p, s * (p < r["experts"])))(*keep["route"](h, v, pre, r)))
    elif what == "scores of real experts only":
        def route(h, w, pre, r):
            picks, _ = keep["route"](h, w, pre, r)
            z = oracle.linear(h, w, pre + "router")
            e = np.exp(z - z.max(-1, keepdims=True))
            s = np.take_along_axis(e, picks, -1)
            return picks, s / s.sum(-1, keepdims=True) * (r["scale"] if r["identity"] == 0 else 1.0)
        patch.setattr(oracle, "route", route)
    elif what == "no limit":
        patch.setattr(oracle, "expert", lambda h, v, pre, limit: keep["expert"](h, v, pre, 1e9))
    elif what == "no plus one":
        patch.setattr(oracle, "expert", lambda h, v, pre, limit: keep["expert"](h, v, pre, limit) - oracle.linear((lambda g: g * oracle.sigmoid(oracle.SLOPE * g))(np.minimum(oracle.linear(h, v, pre + "gate"), limit)), v, pre + "down"))
    elif what == "one cache for all passes":
        def forward(ids, first, w, cfg, caches, residuals=None):
            x = x0 = oracle.embed(ids, w, cfg)
            for i, t in oracle.order(cfg):
                x = oracle.pass_start(x, x0, w, t) if t is not None else x
                n = first + len(ids)
                x = oracle.layer(x, w, i, cfg["layers"][i], cfg["norm"]["eps"], list(range(first, n)), caches[i])
                for name in ("keys", "values", "latents", "parts"):
                    if name in caches[i]:
                        caches[i][name] = caches[i][name][:n]
            return oracle.head(x, w, cfg)
        patch.setattr(oracle, "forward", forward)
    elif what == "one pass less":
        cfg["loop"]["times"] -= 1
    elif what == "x and x0 exchanged":
        patch.setattr(oracle, "pass_start", lambda x, x0, v, t: keep["pass_start"](x0, x, v, t))
    elif what == "the first pass's vector":
        patch.setattr(oracle, "pass_start", lambda x, x0, v, t: keep["pass_start"](x, x0, v, 0))
    elif what == "pass start at the first pass only":
        patch.setattr(oracle, "order", lambda c: [(i, t if t == 0 else None) for i, t in keep["order"](c)])
    elif what == "embedding scale":
        cfg["embedding"]["scale"] = 1.0
    elif what == "logit scale":
        cfg["logit_scale"] = 1.0
    elif what == "eps":
        cfg["norm"]["eps"] = 1e-2
    elif what == "plain sigmoid":
        patch.setattr(oracle, "SLOPE", 1.0)
    elif what == "gelu":
        patch.setattr(oracle, "gelu", lambda z: z * oracle.sigmoid(1.702 * z))
    else:  # a tensor left out
        w[what] = np.ones_like(w[what]) if what.endswith("norm") or what.endswith(("norm1", "norm2")) else np.zeros_like(w[what])


@pytest.mark.parametrize("what", ["window 1 longer", "window 1 shorter", "window 2 longer", "window 2 shorter", "no softcap", "scale 0", "scale 1", "scale 2", "turned halves", "no magnitude", "plain frequencies 0",
                                  "plain frequencies 1", "places from 1", "values after the norm", "norm by head", "taps reversed", "a lost state", "weights with the correction", "choice without the correction",
                                  "identity gives nothing", "scores of real experts only", "no limit", "no plus one", "one cache for all passes", "one pass less", "x and x0 exchanged", "the first pass's vector",
                                  "pass start at the first pass only", "embedding scale", "logit scale", "eps", "plain sigmoid", "gelu", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.o.b", "l1.mix.q.norm", "l1.mix.k.norm",
                                  "l2.mix.dkv.norm", "l0.norm1", "l1.norm2", "final.norm", "l0.mlp.gate.b", "l0.mlp.up.b", "l0.mlp.down.b", "loop.step"])
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
    got = run()
    diff = np.abs(got - want).max() / want.std() if what == "logit scale" else models.error(got, want)
    assert diff > 0.002


def test_no_choice_of_experts_is_a_close_call():
    for name, cfg in models.CONFIGS.items():
        w = models.weights(cfg)
        ids = np.random.default_rng(4).integers(0, cfg["vocab"], 40).tolist()
        seen = []
        keep, oracle.route = oracle.route, lambda h, v, pre, r: seen.append((oracle.linear(h, v, pre + "router"), v[pre + "correction"], r)) or keep(h, v, pre, r)
        try:
            models.Alone(cfg, w)(ids)
        finally:
            oracle.route = keep
        assert seen
        for z, correction, r in seen:
            if r["top"] < len(correction):
                e = np.exp(z - z.max(-1, keepdims=True))
                s = np.sort(e / e.sum(-1, keepdims=True) + correction, -1)[:, ::-1]
                assert ((s[:, r["top"] - 1] - s[:, r["top"]]) / s[:, r["top"] - 1]).min() > 0.004, name


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
    from ferrite_b200 import vunadra
    from ferrite_b200.serve import Engine, Request
    assert vunadra.REWINDS is False
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
