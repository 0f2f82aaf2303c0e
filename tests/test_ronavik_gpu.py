"""Ronavik on the device, through the framework's own loader, forward, caches, engine and command line, against the oracle:
in fp32 (a sharp bound on the design) and in bf16 (the kernels it is served with)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ronavik_models as models
from conftest import ROOT

pytestmark = pytest.mark.gpu

# root mean square of a row's difference over the logits' own: fp32 against float64; bf16 rounds every activation a few
# dozen times on its way through these few layers
BOUND = {"float32": 1e-4, "bfloat16": 0.05, "bfp8": 0.12}


@pytest.fixture(scope="module")
def rt(cuda):
    from ferrite_b200.tensor import Runtime
    return Runtime(0)


@pytest.fixture(scope="module")
def loaded(rt, tmp_path_factory):
    """(name, dtype) -> (config.json, oracle weights, config, device weights), each made once."""
    from ferrite_b200.__main__ import load
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            cfg = models.CONFIGS[name]
            raw = models.weights(cfg)
            _, c, w = load(models.save(tmp_path_factory.mktemp(name), cfg, raw), dtype, 600)
            made[name, dtype] = cfg, raw, c, w
        return made[name, dtype]
    return get


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def replay(rt, loaded, name, dtype, places=400, chunk=2048):
    from ferrite_b200.serve import Replay
    cfg, raw, c, w = loaded(name, dtype)
    return cfg, raw, Replay(rt, w, c, places, chunk)


def on(rt, row):
    from ferrite_b200.tensor import Tensor
    return Tensor.of(rt, [row], "int32")


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_by_layer(rt, loaded, name, dtype):
    from ferrite_b200 import ronavik, llama
    from oracle import ronavik as oracle
    cfg, raw, c, w = loaded(name, dtype)
    ids, want, got = tokens(cfg, 70), [], []
    oracle.forward(ids, 0, raw, cfg, oracle.caches(cfg), want)
    ronavik.forward(on(rt, ids), on(rt, list(range(70))), w, c, ronavik.kv_cache(c, 80, llama.zeros(rt)), residuals=got)
    for i, (a, b) in enumerate(zip(got, want)):
        assert np.abs(a.numpy()[0] - b).max() < (2e-5 if dtype == "float32" else 0.04) * np.abs(b).max(), i


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_prompt_whole_in_portions_and_token_by_token(rt, loaded, name, dtype):
    cfg, raw, run = replay(rt, loaded, name, dtype)
    ids = tokens(cfg, 150)
    want = models.Alone(cfg, raw)(ids)
    got = run.step([("whole", ids, list(range(150)))])
    run.end("whole")
    assert models.error(got, want) < BOUND[dtype]
    # portions: at, before and after the edges of the kernels' tiles and chunks, two tokens and one; each starts in a used slot
    for k, cuts in enumerate(([64, 64, 22], [2] * 5 + [55, 1, 1, 83], [63, 2, 65, 20], [20, 13, 31, 2, 84], [149, 1])):
        at, rows = 0, []
        for n in cuts:
            rows.append(run.step([(f"cut{k}", ids[at:at + n], list(range(n)))]))
            at += n
        run.end(f"cut{k}")
        assert models.error(np.concatenate(rows), want) < BOUND[dtype], cuts
    rows = [run.step([("one", ids[:1], [0])])] + [run.step([("one", [i], [0])]) for i in ids[1:]]
    assert models.error(np.concatenate(rows), want) < BOUND[dtype]


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("mixed", "bfloat16"), ("odd", "float32"), ("odd", "bfloat16"), ("wide", "bfloat16")])
def test_unequal_requests_together_are_each_alone(rt, loaded, name, dtype):
    cfg, raw, run = replay(rt, loaded, name, dtype)
    lengths = [1, 130, 64, 17, 65]
    for turn in range(2):  # (the second time in slots that the first has left)
        ids = [tokens(cfg, n + 40, 10 * turn + i) for i, n in enumerate(lengths)]
        alone = [models.Alone(cfg, raw)(x) for x in ids]
        out = run.step([(f"{turn}{i}", x[:n], [n - 1]) for i, (x, n) in enumerate(zip(ids, lengths))])
        want = np.stack([a[n - 1] for a, n in zip(alone, lengths)])
        assert models.error(out, want) < BOUND[dtype]
        for t in range(40):  # the shorter ones end earlier; the order changes from step to step
            live = [i for i in range(5) if t < 40 - 7 * i]
            live = live[t % len(live):] + live[:t % len(live)]
            out = run.step([(f"{turn}{i}", [ids[i][lengths[i] + t]], [0]) for i in live])
            assert models.error(out, np.stack([alone[i][lengths[i] + t] for i in live])) < BOUND[dtype], (turn, t)
            for i in range(5):
                if t == 40 - 7 * i - 1:
                    run.end(f"{turn}{i}")
    # a request's logits are the same whatever stands beside it, up to rounding of one and the same arithmetic
    x = tokens(cfg, 70, 99)
    one = run.step([("a", x, [69])])
    run.end("a")
    many = run.step([("b", tokens(cfg, 33, 98), []), ("a", x, [69]), ("c", tokens(cfg, 3, 97), [])])
    assert np.abs(one - many).max() <= 1e-5 * np.abs(one).max()


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("mixed", "bfloat16"), ("wide", "bfloat16")])
def test_long_decoding(rt, loaded, name, dtype):
    cfg, raw, run = replay(rt, loaded, name, dtype, places=420)
    ids = tokens(cfg, 400, 5)
    want = models.Alone(cfg, raw)(ids)
    rows = [run.step([("x", ids[:3], [0, 1, 2])])] + [run.step([("x", [i], [0])]) for i in ids[3:]]
    assert models.error(np.concatenate(rows), want) < BOUND[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("l", [0, 1, 2])
def test_the_first_tokens_are_felt_far_away(rt, loaded, l, dtype):
    # two prompts that differ in one token, through one layer: nothing before it feels it; what comes after does, however the prompt is cut
    # and when decoded, as much as the oracle says
    from types import SimpleNamespace as NS
    from ferrite_b200.serve import Replay
    from oracle import ronavik as oracle
    cfg, raw, c, w = loaded("mixed", dtype)
    one = NS(**vars(c) | dict(blocks=c.blocks[l:l + 1], layers=1))
    alone = dict(cfg, layers=cfg["layers"][l:l + 1])
    own = {n.replace(f"l{l}.", "l0.", 1): x for n, x in raw.items() if n.startswith(f"l{l}.")} | {n: raw[n] for n in ("embed", "pos", "final.norm")}
    run, a = Replay(rt, dict(w, _blocks=w["_blocks"][l:l + 1]), one, 300), tokens(cfg, 200, 6)
    for at in (0, 1, 3, 64, 130):
        b = list(a)
        b[at] = (a[at] + 1) % cfg["vocab"]
        want = [oracle.forward(x, 0, own, alone, oracle.caches(alone)) for x in (a, b)]
        for cuts in ([200], [at + 1, 199 - at], [150] + [1] * 50):
            rows = []
            for name, ids in (("a", a), ("b", b)):
                got, first = [], 0
                for n in cuts:
                    got.append(run.step([(name, ids[first:first + n], list(range(n)))]))
                    first += n
                run.end(name)
                rows.append(np.concatenate(got))
                assert models.error(rows[-1], want[len(rows) - 1]) < BOUND[dtype]
            moved = np.abs(rows[0] - rows[1]).max(-1)
            assert (moved[:at] == 0).all() and moved[at] > 0.1
            assert dtype == "bfloat16" or np.abs((rows[0] - rows[1]) - (want[0] - want[1])).max() < 1e-4 * np.abs(want[0]).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_reach_back_over_portions(rt, loaded, dtype):
    # a portion goes on from the states that the one before left, wherever it begins, and a sequence's first tokens from nothing of the
    # sequence that had the slot before
    cfg, raw, run = replay(rt, loaded, "mixed", dtype)
    ids, other = tokens(cfg, 30, 21), tokens(cfg, 30, 22)
    want = models.Alone(cfg, raw)(ids)
    for cuts in ([1, 1, 1, 27], [2, 1, 27], [3, 3, 24], [4, 2, 2, 2, 20], [29, 1]):
        run.step([("before", other, [])])
        run.end("before")
        at, rows = 0, []
        for n in cuts:
            rows.append(run.step([("x", ids[at:at + n], list(range(n)))]))
            at += n
        run.end("x")
        assert models.error(np.concatenate(rows), want) < BOUND[dtype], cuts


def test_block_floats(rt, loaded, tmp_path):
    from ferrite_b200.__main__ import load
    from ferrite_b200.serve import Replay
    cfg = models.config(128, 160, [models.mamba2(heads=16, vdim=16, state=32, mlp=models.moe(ff=64), norm_groups=2), models.parallel(heads=4, kv_heads=2, dim=32, vdim=48, mlp=models.moe(ff=64)), models.mamba2(mlp=None)])
    raw = models.weights(cfg)
    _, c, w = load(models.save(tmp_path, cfg, raw), "bfp8", 300)
    assert w["l0.in"].dtype == w["l1.in"].dtype == w["l1.mix.o"].dtype == w["head"].dtype == "bfp8"
    assert w["l1.mlp.in"].dtype == w["l1.mlp.up"].dtype == w["l1.mix.gates"].dtype == w["l2.in"].dtype == "bf16"
    run, ids = Replay(rt, w, c, 220), tokens(cfg, 200, 6)
    want = models.Alone(cfg, raw)(ids)
    got = np.concatenate([run.step([("x", ids[:150], list(range(150)))])] + [run.step([("x", ids[150:190], list(range(40)))])] + [run.step([("x", [i], [0])]) for i in ids[190:]])
    assert models.error(got, want) < BOUND["bfp8"]


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("odd", "float32"), ("wide", "bfloat16")])
def test_greedy_generation_by_the_engine(rt, loaded, name, dtype):
    from ferrite_b200.serve import DeviceBackend, Engine, Request
    cfg, raw, c, w = loaded(name, dtype)
    system = tokens(cfg, 20, 7)
    prompts = [system + [3, 4], tokens(cfg, 70, 8), system + [5], tokens(cfg, 1, 9), tokens(cfg, 33, 10)]
    engine = Engine(DeviceBackend(rt, w, c, 2, 120), 2, 120, chunk=24)
    for r in engine.run([Request(p, max_tokens=8 + i) for i, p in enumerate(prompts)]):
        run, at = models.Alone(cfg, raw), 0
        out = run(r.ids)
        for t in r.made:  # teacher-forced by the engine's own picks: each is the oracle's unless the best two are as good as equal
            best = out[-1].max()
            assert best - out[-1][t] <= (1e-3 if dtype == "float32" else 0.15) * out[-1].std(), (len(r.ids), at, t)
            out, at = run([t]), at + 1
        assert r.finish == "length" and len(r.made) == r.max_tokens
    if dtype == "float32":  # a slot all of which begins a prompt goes on from there, one of which only a part does starts anew
        for ids, cached in ((engine.held[0] + [1, 2], len(engine.held[0])), (engine.held[1][:-3] + [1], 0)):
            r = Request(ids, max_tokens=3)
            engine.run([r])
            assert r.cached == cached and r.made == models.greedy(cfg, raw, r.ids, 3)
    sampled = [Engine(DeviceBackend(rt, w, c, 2, 60), 2, 60).run([Request(prompts[0], 6, temperature=0.8, top_k=10, seed=4)])[0].made for _ in range(2)]
    assert sampled[0] == sampled[1] and len(sampled[0]) == 6


def test_a_recorded_step_is_the_eager_step(rt, loaded):
    cfg, raw, c, w = loaded("mixed", "bfloat16")
    from ferrite_b200 import ronavik, llama
    from ferrite_b200.tensor import jit
    rows = []
    for wrap in (jit, lambda f: f):
        kv = ronavik.kv_cache(c, 2 * 40, llama.zeros(rt), 2)
        step = wrap(lambda ids, at: ronavik.forward(ids, at, w, c, kv, 2).realize())
        rows.append([step(on(rt, [5 + i, 90 - i]), on(rt, [i, i])).numpy().copy() for i in range(30)])
    assert all(np.array_equal(a, b) for a, b in zip(*rows))


def test_random_weights_run(rt):
    from ferrite_b200 import ronavik, llama
    c = ronavik.config(models.CONFIGS["mixed"], 100)
    for mode in ("bf16", "fp32"):
        c, prec = ronavik.with_precision(c, mode)
        w = ronavik.random_weights(rt, c, prec)
        kv = ronavik.kv_cache(c, 50, llama.zeros(rt))
        assert np.isfinite(ronavik.forward(on(rt, [1, 2, 3]), on(rt, [0, 1, 2]), w, c, kv, every=True).numpy()).all()


def test_command_line(rt, tmp_path):
    cfg = models.CONFIGS["mixed"]
    raw = models.weights(cfg, 3)
    folder = models.save(tmp_path / "model", cfg, raw)
    a, b = tokens(cfg, 12, 11), tokens(cfg, 5, 12)
    out = subprocess.run([sys.executable, "-m", "ferrite_b200", "generate", "--model", folder, "--dtype", "float32", "--max-tokens", "6",
                          "--ids", ",".join(map(str, a)), "--ids", ",".join(map(str, b))], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    lines = [json.loads(line) for line in out.stdout.splitlines()]
    assert [line["prompt"] for line in lines] == [a, b] and all(line["tokens"] == models.greedy(cfg, raw, line["prompt"], 6) for line in lines)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": a, "want": [3, 11]}, {"id": "q", "tokens": b, "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": [8], "want": [0]}, {"id": "p", "tokens": [9], "want": [0]}], "end": ["p", "q"]},
             {"step": 2, "entries": [{"id": "r", "tokens": b, "want": []}], "end": ["r"]}]
    for dtype in ("float32", "bfloat16"):
        folder_out = tmp_path / dtype
        folder_out.mkdir()
        out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(folder_out), "--max-tokens", "40"],
                             input="".join(json.dumps(s) + "\n" for s in steps), cwd=tmp_path, capture_output=True, text=True, timeout=300)
        assert out.returncode == 0, out.stderr
        assert [line for line in out.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
        got = [np.fromfile(folder_out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in range(2)]
        p, q = models.Alone(cfg, raw)(a + [9]), models.Alone(cfg, raw)(b + [8])
        assert models.error(got[0], p[[3, 11]]) < BOUND[dtype] and models.error(got[1], np.stack([q[5], p[12]])) < BOUND[dtype]
        assert not (folder_out / "2.f32").exists()
