"""The command line.

    python -m ferrite_b200 generate --model DIR --ids 5,17,3 [--ids ...] [--max-tokens N] [--temperature T] [--slots S]
    python -m ferrite_b200 replay --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   (bin/trace_run)

`generate` decodes token ids with the slot engine (there is no tokenizer here) and prints a JSON line a request.  `replay`
feeds given tokens through the same device side: it reads steps from standard input, a JSON object a line with `step`,
`entries` (each an `id`, its next `tokens`, and `want`, the places among them whose logits are asked for) and `end` (the
requests that are finished after it), writes the wanted logits to OUT/<step>.f32 (little-endian fp32, [wanted, vocabulary])
and prints `done <step>`."""
import argparse
import json
import os
import sys

MODES = {"bfloat16": "bf16", "float32": "fp32", "bfp8": "bfp8", "bfp4": "bfp4"}


def load(folder, dtype, places):
    """A runtime, a checkpoint's config and its weights on the device."""
    from . import build, checkpoint, models
    from .tensor import Runtime
    build.ensure(models.family_of_json(checkpoint.read_json(os.path.join(folder, "config.json"))), MODES[dtype])  # (where it is missing)
    rt = Runtime(0)
    c, w = checkpoint.load(folder, places)
    family = models.of(c)
    if hasattr(family, "with_precision"):
        c, prec = family.with_precision(c, MODES[dtype])
    else:
        assert dtype != "float32", f"the {c.family} family keeps its activations in bf16"
        prec = family.precision(c, MODES[dtype])
    return rt, c, family.upload(rt, w, prec)


def generate(a):
    from .serve import DeviceBackend, Engine, Request
    prompts = [[int(v) for v in text.split(",")] for text in a.ids]
    places = max(map(len, prompts)) + a.max_tokens + 2
    rt, c, w = load(a.model, a.dtype, places)
    engine = Engine(DeviceBackend(rt, w, c, a.slots, places), a.slots, places, a.chunk)
    for r in engine.run([Request(p, a.max_tokens, a.temperature, a.top_k, seed=a.seed) for p in prompts]):
        print(json.dumps({"prompt": r.ids, "tokens": r.made, "finish": r.finish}), flush=True)
    return 0


def replay(a):
    from .serve import Replay
    rt, c, w = load(a.model, a.dtype, a.max_tokens + 2)
    run = Replay(rt, w, c, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = run.step([(e["id"], e["tokens"], e["want"]) for e in s["entries"]]) if s["entries"] else None
        if out is not None:
            out.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        else:
            rt.wait()
        for name in s["end"]:
            run.end(name)
        print(f"done {s['step']}", flush=True)
    return 0


def main(args=None):
    ap = argparse.ArgumentParser(prog="ferrite_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g, r = sub.add_parser("generate"), sub.add_parser("replay")
    for p in (g, r):
        p.add_argument("--model", required=True, help="a folder with config.json and model.safetensors")
    g.add_argument("--dtype", default="bfloat16", choices=sorted(MODES))
    g.add_argument("--ids", action="append", required=True, help="a prompt's token ids, with commas (once a request)")
    g.add_argument("--max-tokens", type=int, default=16)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--seed", type=int, default=None)
    g.add_argument("--slots", type=int, default=4)
    g.add_argument("--chunk", type=int, default=512, help="tokens of a prompt that go in at once")
    r.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    r.add_argument("--out", required=True)
    r.add_argument("--max-tokens", type=int, default=4096, help="the most tokens that live requests hold together")
    a = ap.parse_args(args)
    return generate(a) if a.command == "generate" else replay(a)


if __name__ == "__main__":
    sys.exit(main())
