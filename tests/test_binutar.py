"""Binutar on the host: its configuration and checkpoint as the loader reads them, the oracle against itself however a
sequence is cut, what the tests' weights let through, and the slot engine over a backend whose state cannot be taken back."""
import copy
import json
from types import SimpleNamespace as NS

import numpy as np
import pytest

import binutar_models as models
from oracle import binutar as oracle


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
def test_a_checkpoint_loads_by_its_config(tmp_path, name):
    from ferrite_b200 import binutar, checkpoint, models as registry
    cfg = models.CONFIGS[name]
    raw = models.weights(cfg)
    c, w = checkpoint.load(models.save(tmp_path, cfg, raw), places=77)
    assert registry.of(c) is binutar and (c.family, c.dim, c.vocab, c.layers, c.places, c.eps) == ("binutar", cfg["width"], cfg["vocab"], len(cfg["layers"]), 77, cfg["norm"]["eps"])
    for i, e in enumerate(cfg["layers"]):
        m, p = c.blocks[i].mixer, f"l{i}."
        assert (c.blocks[i].type, m.heads, m.dim, m.vdim) == (e["type"], *(e["mixer"][k] for k in ("heads", "dim", "vdim")))
        if e["type"] == "latent_attention":
            assert np.array_equal(w[p + "mix.in"].values(), np.concatenate([raw[p + "mix." + n] for n in ("dq", "dkv", "g")]).T)
            assert np.array_equal(w[p + "mix.uk"].values(), raw[p + "mix.uk"].reshape(m.heads, m.dim, m.kv_rank))
            assert np.array_equal(w[p + "mix.uv"].values(), raw[p + "mix.uv"].reshape(m.heads, m.vdim, m.kv_rank).swapaxes(1, 2))
        else:
            assert np.array_equal(w[p + "mix.qkvg"].values(), np.concatenate([raw[p + "mix." + n] for n in "qkvg"]).T)
        assert (p + "mlp.gate_up" in w) == bool(e["mlp"])
    assert np.array_equal(w["head"].values(), raw["head"].T) and w["l0.norm1.alpha"].values().size == 1
    fmt = binutar.precision(c, "bf16")
    assert binutar.weight_format("l0.norm1", fmt) == binutar.weight_format("final.norm.alpha", fmt) == "fp32" and binutar.weight_format("l0.mix.o", fmt) == "bf16"
    assert binutar.weight_format("embed", binutar.precision(c, "fp32")) == binutar.weight_format("l0.mix.uk", binutar.precision(c, "fp32")) == "fp32"


def test_what_is_not_served_is_refused_by_name(tmp_path):
    from ferrite_b200 import binutar, models as registry
    with pytest.raises(AssertionError, match="Nonesuch"):
        registry.of_json({"architecture": "Nonesuch"})
    cfg = copy.deepcopy(models.CONFIGS["turns"])
    cfg["layers"][1]["type"] = "stroll"
    with pytest.raises(AssertionError, match="stroll"):
        binutar.config(cfg)
    cfg = copy.deepcopy(models.CONFIGS["turns"])
    cfg["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(AssertionError, match="sparse"):
        binutar.config(cfg)
    cfg = copy.deepcopy(models.CONFIGS["turns"])
    cfg["layers"][1]["mixer"]["decay"].pop()
    with pytest.raises(AssertionError, match="a decay a head"):
        binutar.config(cfg)


@pytest.mark.parametrize("scaling", [None, dict(factor=4.0, original=2000, fast=30.0, slow=1.0), dict(factor=2.0, original=64, fast=3.0, slow=2.9), dict(factor=8.0, original=100000, fast=2.0, slow=0.5)])
@pytest.mark.parametrize("dims,base", [(32, 10000.0), (2, 500.0), (64, 50.0)])
def test_frequencies(scaling, dims, base):
    from ferrite_b200 import mixers
    want, mag = oracle.yarn(dict(dims=dims, base=base, scaling=scaling))
    got, factor = mixers.frequencies(NS(dims=dims, base=base, scaling=NS(**scaling) if scaling else None))
    np.testing.assert_allclose(got, want, rtol=1e-12)
    assert factor == pytest.approx(mag)


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


@pytest.mark.parametrize("what", ["sink", "decay", "scale", "limit", "factor", "place", "first token"])
def test_the_weights_show_a_mistake(what):
    # planted in the oracle: each is far above what the tests allow the device in fp32
    cfg = copy.deepcopy(models.CONFIGS["turns"])
    w = models.weights(cfg)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 40).tolist()
    want = models.Alone(cfg, w)(ids)
    m0, first, start = cfg["layers"][0]["mixer"], list(ids), 0
    if what == "sink":
        w["l0.mix.sink"] = np.full_like(w["l0.mix.sink"], -np.inf)
    elif what == "decay":
        cfg["layers"][1]["mixer"]["decay"][2] = 0.98
    elif what == "scale":
        m0["scale"] *= 1.02
    elif what == "limit":
        cfg["layers"][1]["mlp"]["limit"] = 1.0
    elif what == "factor":
        m0["rot"]["scaling"]["factor"] = 2.7
    elif what == "place":
        m0["rot"]["base"] *= 1.5
    else:
        first[0] = (first[0] + 1) % cfg["vocab"]
    assert models.error(models.Alone(cfg, w)(first)[1:], want[1:]) > 0.002


class OracleBackend:
    """The engine's device side played by the oracle: a slot's state starts anew when its first token stands at place 0."""
    rewinds = False

    def __init__(self, cfg, w, slots):
        self.cfg, self.w, self.caches, self.prefills = cfg, w, [oracle.caches(cfg) for _ in range(slots)], []

    def head(self, logits):
        order = np.argsort(-logits, kind="stable")[:64]
        return logits[order], order, 0.0

    def run(self, u, ids, first):
        if first == 0:
            self.caches[u] = oracle.caches(self.cfg)
        return self.head(oracle.forward(ids, first, self.w, self.cfg, self.caches[u])[-1])

    def prefill(self, u, ids, first, t):
        self.prefills.append((u, first, len(ids)))
        return self.run(u, ids, first)

    def decode(self, ids, places, ts):
        return [self.run(u, [i], p) if p < 63 else None for u, (i, p) in enumerate(zip(ids, places))]


def test_engine_reuses_a_slot_only_from_where_its_state_stands():
    from ferrite_b200.serve import Engine, Request
    cfg = models.CONFIGS["linear"]
    w = models.weights(cfg)
    rng = np.random.default_rng(3)
    draw = lambda n: rng.integers(0, cfg["vocab"], n).tolist()
    system = draw(9)
    backend = OracleBackend(cfg, w, 2)
    engine = Engine(backend, slots=2, places=64, chunk=4)
    first = engine.run([Request(system + [3, 4], max_tokens=5)])[0]
    held = system + [3, 4] + first.made[:-1]
    rs = engine.run([Request(p, max_tokens=6) for p in (held + [7, 8], system + [3, 4], system + [5], held + [7], draw(3))])
    assert rs[0].cached == len(held), "the whole of what the slot holds begins the prompt"
    assert rs[1].cached == rs[2].cached == 0, "a part of it is of no use to a recurrent state"
    for r in [first, *rs]:
        want, _ = models.greedy(cfg, w, r.ids, r.max_tokens)
        assert r.made == want and r.finish == "length"
    assert all(n <= 4 for _, _, n in backend.prefills)


def test_replay_deals_out_slots(monkeypatch):
    from ferrite_b200 import serve

    class Backend:
        def __init__(self, rt, w, c, slots, places):
            self.slots, self.part, self.calls = slots, places, []

        def prompt(self, u, ids, first, every=False):
            self.calls.append(("prompt", u, list(ids), first))
            rows = np.array([[float(u), float(first + i)] for i in (every or [0])], np.float32)
            return NS(numpy=lambda: rows[None])

        def token(self, ids, places):
            self.calls.append(("token", list(ids), list(places)))
            return NS(numpy=lambda: np.array([[float(u), float(p)] for u, p in enumerate(places)], np.float32)[None])
    monkeypatch.setattr(serve, "DeviceBackend", Backend)
    r = serve.Replay(None, None, None, places=20, chunk=4)
    out = r.step([("a", [1, 2, 3, 4, 5, 6], [0, 4, 5]), ("b", [9], [])])
    assert out.tolist() == [[0, 0], [0, 4], [0, 5]] and [c[3] for c in r.backend.calls] == [0, 4, 0]
    out = r.step([("b", [7], [0]), ("a", [8], [0])])
    assert out.tolist() == [[1, 1], [0, 6]] and r.backend.calls[-1] == ("token", [8, 7], [6, 1])
    r.end("a")
    assert r.step([("b", [7], [])]) is None and r.backend.calls[-1] == ("token", [0, 7], [21, 2]), "a free slot's token stands at the last place"
    backend = r.backend
    r.end("b")
    r.step([("c", [1, 2], [1])])
    assert r.backend is backend and r.slot == {"c": 0} and r.backend.calls[-1][3] == 0
    with pytest.raises(AssertionError, match="every slot is taken"):
        r.step([("d", [1], []), ("e", [1], [])])


def test_command_line_asks_for_a_model():
    from ferrite_b200.__main__ import main
    with pytest.raises(SystemExit):
        main(["replay"])
    with pytest.raises(SystemExit):
        main(["replay", "--model", "x", "--out", "y", "--dtype", "float16"])
    json.dumps(models.CONFIGS)  # (a config is plain JSON)


def test_the_library_is_built_for_a_family_and_completed_later(tmp_path, monkeypatch):
    # the compiler played by a function that writes files: which sources are compiled and linked, and when
    from ferrite_b200 import build
    for name, at in (("OBJ", "obj"), ("LIB", "lib/lib.so"), ("LINKED", "lib/sources.txt")):
        monkeypatch.setattr(build, name, str(tmp_path / at))
    compiled, linked = [], []

    def compile_one(name):
        compiled.append(name)
        return name, ""

    def run(cmd, **_):
        linked.append([o.split("/")[-1] for o in cmd if o.endswith(".o")])
        open(build.LIB, "w").close()
        return NS(returncode=0, stdout="", stderr="")
    monkeypatch.setattr(build, "compile_one", compile_one)
    monkeypatch.setattr(build.subprocess, "run", run)
    need = build.FAMILY_SOURCES["binutar"]
    assert set(need) < set(build.sources())
    build.ensure("binutar")
    assert sorted(compiled) == sorted(need) and len(linked[-1]) == len(need) and build.linked() == sorted(need)
    build.ensure("binutar", "fp32")
    assert len(linked) == 1, "nothing is missing"
    build.ensure("binutar", "bfp8")
    assert len(linked) == 2 and len(linked[-1]) == len(build.sources()) and build.linked() == build.sources()
    build.ensure("llama")
    build.ensure("binutar")
    assert len(linked) == 2
