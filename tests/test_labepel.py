"""Labepel on the host: its configuration and checkpoint as the loader reads them, the oracle against itself however a sequence
is cut, mistakes planted in the oracle (each must show), the slot engine over a backend played by the oracle."""
import copy

import numpy as np
import pytest

import labepel_models as models
from oracle import labepel as oracle


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
def test_a_checkpoint_loads_by_its_config(tmp_path, name):
    from ferrite_b200 import checkpoint, labepel, models as registry
    cfg = models.CONFIGS[name]
    raw = models.weights(cfg)
    c, w = checkpoint.load(models.save(tmp_path, cfg, raw), places=77)
    assert registry.of(c) is labepel
    assert (c.family, c.dim, c.vocab, c.layers, c.places, c.eps, c.positions) == ("labepel", cfg["width"], cfg["vocab"], len(cfg["layers"]), 77, cfg["norm"]["eps"], cfg["max_positions"])
    fmt, exact = labepel.precision(c, "bf16"), labepel.precision(c, "fp32")
    for i, e in enumerate(cfg["layers"]):
        m, p = c.blocks[i].mixer, f"l{i}."
        assert (m.heads, m.kv_heads, m.dim, m.vdim, m.mask.size, m.scale, m.v_mix) == tuple(e["mixer"][k] if k != "mask" else e["mixer"]["mask"]["size"]
                                                                                         for k in ("heads", "kv_heads", "dim", "vdim", "mask", "scale", "v_mix"))
        assert np.array_equal(w[p + "in"].values(), np.concatenate([raw[p + "mix." + n] for n in "qkvg"]))
        assert np.array_equal(w[p + "mix.b"].values()[0], np.concatenate([raw[p + "mix." + n + ".b"] for n in "qkv"]))
        assert (p + "mlp.gate_up" in w) == bool(e["mlp"]) and (p + "mlp.shared.down" in w) == bool(e["mlp"] and e["mlp"].get("shared"))
        if e["mlp"]:
            last = e["mlp"]["router"]["experts"] - 1
            assert w[p + "mlp.gate_up"].values().shape == (last + 1, cfg["width"], 2 * e["mlp"]["expert"]["ff"])
            assert np.array_equal(w[p + "mlp.gate_up"].values()[last], np.concatenate([raw[f"{p}mlp.e{last}.gate"], raw[f"{p}mlp.e{last}.up"]]).T)
            assert np.array_equal(w[p + "mlp.down"].values()[last], raw[f"{p}mlp.e{last}.down"].T)
        for n in ("norm1", "ls1", "mix.b", "mix.q.norm", "mix.vmix", "mlp.router.b"):
            assert labepel.weight_format(p + n, fmt) == "fp32"
        assert labepel.weight_format(p + "in", fmt) == labepel.weight_format(p + "mlp.down", fmt) == "bf16" and labepel.weight_format(p + "mlp.down", exact) == "fp32"
    assert labepel.weight_format("pos", fmt) == "bf16" and labepel.weight_format("head", exact) == labepel.weight_format("embed", exact) == "fp32"


def test_block_float_formats_leave_the_router_alone():
    from ferrite_b200 import labepel
    c = labepel.config(models.CONFIGS["mixed"])
    prec = labepel.precision(c, "bfp8")
    assert labepel.weight_format("l0.mix.o", prec) == labepel.weight_format("l0.mlp.down", prec) == "bfp8"
    assert labepel.routed_apart(0, prec) and labepel.weight_format("l0.mlp.router", prec) == "bf16" and not labepel.routed_apart(0, labepel.precision(c))
    odd = labepel.precision(labepel.config(models.CONFIGS["odd"]), "bfp8")
    assert odd["in", 1][0] == odd["mlp.gate_up", 0][0] == odd["mlp.down", 0][0] == "bf16", "no whole runs of 16 columns"


@pytest.mark.parametrize("change,what", [(lambda e: e.update(type="stroll"), "stroll"), (lambda e: e["mlp"].update(kind="dense"), "dense"), (lambda e: e["mixer"].update(kv_heads=3), "whole groups"),
                                         (lambda e: e["mlp"]["router"].update(top=9), "9 of 6"), (lambda e: e["mixer"].update(v_mix=True, vdim=36), "as wide")])
def test_what_is_not_served_is_refused_by_name(change, what):
    from ferrite_b200 import labepel
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    change(cfg["layers"][3])
    if what == "9 of 6":
        cfg["layers"][3]["mlp"]["router"]["experts"] = 6
    with pytest.raises(AssertionError, match=what):
        labepel.config(cfg)


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
    m = cfg["layers"][1]["mixer"]
    keep = {n: getattr(oracle, n) for n in ("attend", "mix_values", "route", "sigmoid", "layer")}
    if what == "a span one longer":
        m["mask"]["size"] += 1
    elif what == "a span one shorter":
        m["mask"]["size"] -= 1
    elif what == "a span that begins a key late":
        patch.setattr(oracle, "chunk_of", lambda place, size: min(place, place // size * size + 1))
    elif what == "a window for a span":
        patch.setattr(oracle, "chunk_of", lambda place, size: max(0, place - size + 1))
    elif what == "no sink":
        patch.setattr(oracle, "attend", lambda q, k, v, places, size, scale: keep["attend"](q, k, np.concatenate([v, np.ones_like(v[..., :1])], -1), places, size, scale)[..., :-1]
                      / keep["attend"](q, k, np.concatenate([v, np.ones_like(v[..., :1])], -1), places, size, scale)[..., -1:])
    elif what == "values not mixed":
        patch.setattr(oracle, "mix_values", lambda v, first, share: v)
    elif what == "mixed with the layer before":
        def layer(x, w, i, entry, eps, places, cache, shared):
            out = keep["layer"](x, w, i, entry, eps, places, cache, shared)
            if entry["mixer"].get("v_mix"):
                shared["v"] = cache["v"][-len(places):]
            return out
        patch.setattr(oracle, "layer", layer)
    elif what == "weights before the choice":
        def route(h, w, pre, m):
            picks, _ = keep["route"](h, w, pre, m)
            z = h @ w[pre + "router"].T + w[pre + "router.b"]
            e = np.exp(z - z.max(-1, keepdims=True))
            return picks, np.take_along_axis(e / e.sum(-1, keepdims=True), picks, -1)
        patch.setattr(oracle, "route", route)
    elif what in ("mix.q.b", "mix.k.b", "mix.v.b", "mlp.router.b", "mix.g", "mlp.shared.down"):
        w["l1." + what] = np.zeros_like(w["l1." + what])
    elif what in ("mix.q.norm", "mix.k.norm", "ls1", "ls2"):
        w["l1." + what] = np.ones_like(w["l1." + what])
    elif what == "norm1":
        w["l1.norm1"] = w["l1.norm1"] - 1
    elif what == "scale":
        m["scale"] *= 1.02
    elif what == "places":
        w["pos"] = np.roll(w["pos"], 1, 0)
    elif what == "eps":
        cfg["norm"]["eps"] = 1e-2


@pytest.mark.parametrize("what", ["a span one longer", "a span one shorter", "a span that begins a key late", "a window for a span", "no sink", "values not mixed", "mixed with the layer before",
                                  "weights before the choice", "mix.q.b", "mix.k.b", "mix.v.b", "mlp.router.b", "mix.g", "mlp.shared.down", "mix.q.norm", "mix.k.norm", "ls1", "ls2", "norm1",
                                  "scale", "places", "eps"])
def test_the_weights_show_a_mistake(what, monkeypatch):
    # each is far above what the tests allow the device in fp32
    cfg = copy.deepcopy(models.CONFIGS["mixed"])
    if what in ("mixed with the layer before", "values not mixed"):
        cfg["layers"] = [models.attention() for _ in range(3)]
    w = models.weights(cfg)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 80).tolist()
    want = models.Alone(cfg, w)(ids)
    planted(what, cfg, w, monkeypatch)
    assert models.error(models.Alone(cfg, w)(ids), want) > 0.002


def test_no_choice_of_experts_is_a_close_call():
    for name, cfg in models.CONFIGS.items():
        w = models.weights(cfg)
        ids = np.random.default_rng(4).integers(0, cfg["vocab"], 60).tolist()
        res = []
        oracle.forward(ids, 0, w, cfg, oracle.caches(cfg), res)
        x = np.float64(w["embed"])[ids] + w["pos"][:60]
        for i, e in enumerate(cfg["layers"]):
            if e["mlp"] and e["mlp"]["router"]["top"] < e["mlp"]["router"]["experts"]:
                h = oracle.rms(x, 1 + np.float64(w[f"l{i}.norm1"]), cfg["norm"]["eps"])
                z = np.sort(h @ w[f"l{i}.mlp.router"].T + w[f"l{i}.mlp.router.b"], -1)[:, ::-1]
                k = e["mlp"]["router"]["top"]
                assert (z[:, k - 1] - z[:, k]).min() > 0.01 * np.abs(z).max(), (name, i)
            x = res[i]


class OracleBackend:
    """The engine's device side played by the oracle; what a slot holds past a prompt's place is overwritten (rewinds)."""

    def __init__(self, cfg, w, slots):
        self.cfg, self.w, self.caches = cfg, w, [oracle.caches(cfg) for _ in range(slots)]

    def head(self, logits):
        order = np.argsort(-logits, kind="stable")[:64]
        return logits[order], order, 0.0

    def run(self, u, ids, first):
        for cache in self.caches[u]:
            for name in cache:
                cache[name] = cache[name][:first]
        return self.head(oracle.forward(ids, first, self.w, self.cfg, self.caches[u])[-1])

    def prefill(self, u, ids, first, t):
        return self.run(u, ids, first)

    def decode(self, ids, places, ts):
        return [self.run(u, [i], p) if p < 63 else None for u, (i, p) in enumerate(zip(ids, places))]


def test_engine_goes_on_from_a_prefix_that_a_slot_still_holds():
    from ferrite_b200.serve import Engine, Request
    cfg = models.CONFIGS["mixed"]
    w = models.weights(cfg)
    rng = np.random.default_rng(3)
    draw = lambda n: rng.integers(0, cfg["vocab"], n).tolist()
    system = draw(9)
    engine = Engine(OracleBackend(cfg, w, 2), slots=2, places=64, chunk=4)
    rs = engine.run([Request(system + [3, 4], max_tokens=5)]) + engine.run([Request(p, max_tokens=6) for p in (system + [5], draw(3), system + [3, 4, 8])])
    assert rs[1].cached == 9 and all(r.made == models.greedy(cfg, w, r.ids, r.max_tokens) for r in rs)
