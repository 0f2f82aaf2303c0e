"""Binutar on the device, through the framework's own loader, forward, caches, engine and command line, against the oracle:
in fp32 (a sharp bound on the design) and in bf16 (the kernels it is served with)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import binutar_models as models
from conftest import ROOT

pytestmark = pytest.mark.gpu

# root mean square of a row's difference over the logits' own: fp32 against float64; bf16 rounds every activation a few
# dozen times on its way through these few layers
BOUND = {"float32": 2e-4, "bfloat16": 0.06, "bfp8": 0.12}


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


@pytest.mark.parametrize("name", sorted(models.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_prompt_whole_in_portions_and_token_by_token(rt, loaded, name, dtype):
    cfg, raw, run = replay(rt, loaded, name, dtype)
    ids = tokens(cfg, 150)
    want = models.Alone(cfg, raw)(ids)
    got = run.step([("whole", ids, list(range(150)))])
    run.end("whole")
    assert models.error(got, want) < BOUND[dtype]
    # portions: whole tiles of the kernels, across their edges, two tokens and one; each starts in a used slot
    for k, cuts in enumerate(([64, 64, 22], [2] * 5 + [55, 1, 1, 83], [63, 2, 65, 20], [149, 1])):
        at, rows = 0, []
        for n in cuts:
            rows.append(run.step([(f"cut{k}", ids[at:at + n], list(range(n)))]))
            at += n
        run.end(f"cut{k}")
        assert models.error(np.concatenate(rows), want) < BOUND[dtype], cuts
    rows = [run.step([("one", ids[:1], [0])])] + [run.step([("one", [i], [0])]) for i in ids[1:]]
    assert models.error(np.concatenate(rows), want) < BOUND[dtype]


@pytest.mark.parametrize("name,dtype", [("turns", "float32"), ("turns", "bfloat16"), ("odd", "bfloat16"), ("wide", "bfloat16")])
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
            on = [i for i in range(5) if t < 40 - 7 * i]
            on = on[t % len(on):] + on[:t % len(on)]
            out = run.step([(f"{turn}{i}", [ids[i][lengths[i] + t]], [0]) for i in on])
            assert models.error(out, np.stack([alone[i][lengths[i] + t] for i in on])) < BOUND[dtype], (turn, t)
            for i in range(5):
                if t == 40 - 7 * i - 1:
                    run.end(f"{turn}{i}")
    # a request's logits are the same whatever stands beside it, up to rounding of one and the same arithmetic
    x = tokens(cfg, 70, 99)
    one = run.step([("a", x, [69])])
    run.end("a")
    many = run.step([("b", tokens(cfg, 33, 98), []), ("a", x, [69]), ("c", tokens(cfg, 3, 97), [])])
    assert np.abs(one - many).max() <= 1e-5 * np.abs(one).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_far_keys(rt, loaded, dtype):
    cfg, raw, run = replay(rt, loaded, "turns", dtype, places=420)
    ids = tokens(cfg, 400, 5)
    want = models.Alone(cfg, raw)(ids)
    rows = [run.step([("x", ids[:3], [0, 1, 2])])] + [run.step([("x", [i], [0])]) for i in ids[3:]]
    assert models.error(np.concatenate(rows), want) < BOUND[dtype]


def test_block_float_projections(rt, loaded):
    cfg, raw, c, w = loaded("wide", "bfp8")
    assert w["l0.mix.o"].dtype == w["l1.mix.qkvg"].dtype == "bfp8" and w["l0.mix.uk"].dtype == "bf16"
    assert w["l0.mix.in"].cols % 16 and w["l0.mix.in"].dtype == "bf16", "no whole runs of 16 columns: not a block float"
    from ferrite_b200.serve import Replay
    run, ids = Replay(rt, w, c, 100), tokens(cfg, 60, 6)
    want = models.Alone(cfg, raw)(ids)
    got = np.concatenate([run.step([("x", ids[:50], list(range(50)))])] + [run.step([("x", [i], [0])]) for i in ids[50:]])
    assert models.error(got, want) < BOUND["bfp8"]


@pytest.mark.parametrize("name,dtype", [("turns", "float32"), ("linear", "float32"), ("wide", "bfloat16")])
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
    if dtype == "float32":  # a slot whose whole content begins a prompt goes on from there
        held = engine.held[0]
        r = Request(held + [1], max_tokens=3)
        engine.run([r])
        assert r.cached == len(held) and r.made == models.greedy(cfg, raw, r.ids, 3)[0]
    sampled = [Engine(DeviceBackend(rt, w, c, 2, 60), 2, 60).run([Request(prompts[0], 6, temperature=0.8, top_k=10, seed=4)])[0].made for _ in range(2)]
    assert sampled[0] == sampled[1] and len(sampled[0]) == 6


def test_command_line(rt, tmp_path):
    cfg = models.CONFIGS["turns"]
    raw = models.weights(cfg, 3)
    folder = models.save(tmp_path / "model", cfg, raw)
    a, b = tokens(cfg, 12, 11), tokens(cfg, 5, 12)
    out = subprocess.run([sys.executable, "-m", "ferrite_b200", "generate", "--model", folder, "--dtype", "float32", "--max-tokens", "6",
                          "--ids", ",".join(map(str, a)), "--ids", ",".join(map(str, b))], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    lines = [json.loads(line) for line in out.stdout.splitlines()]
    assert [line["prompt"] for line in lines] == [a, b] and all(line["tokens"] == models.greedy(cfg, raw, line["prompt"], 6)[0] for line in lines)
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
