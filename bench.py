"""Decode throughput of the block-float hot path on B200s, one JSON line.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--workload llama8b|smollm] [--layers L] [--impl reference]
    python bench.py --matmul 32,4096,14336,bfp8,6      (one isolated matmul, a few calls: what the ncu captures run)
    python bench.py --attend 32,32,8,128,2048,6        (the decode attention alone, likewise)
    python bench.py --design binutar|labepel|vunadra|ronavik   (prefill, decode and kernels of that design beside the Llama decoder)

The default workload is the Llama-3.1-8B-shape batched decode (32 sequences, 2048 tokens of context each, bfp8 weights,
bf16 KV cache), tensor-parallel over N GPUs with an NCCL all-reduce after o_proj and down_proj.  A step is one decode
step of all the sequences: embedding gather, 32 blocks (fused RMSNorm + qkv matmul, RoPE + KV write, split-KV attention,
o_proj + residual, RMSNorm + gate_up + SwiGLU, down_proj + residual), final norm, output layer, greedy pick.

    value      tokens/s with the step's inputs resident on the device (the pick of one step feeds the next on the device)
    e2e        the same through the public call with host buffers: ids and places copied in from pinned memory and the
               picked tokens read back, every step
    roofline   the block-float matmul kernel (the dominant kernel): its algorithmic bytes over its measured duration
    matmul_sweep  (1 GPU) the isolated matmul with fused RMSNorm and SwiGLU over M, N and both formats: GB/s and fraction of peak
    cpu_baseline / --impl reference: the numpy restatement of the reference's CPU path on this box's host cores, on a
               bounded sample (one block and the output layer, scaled to the model)
"""
import argparse
import json
import os
import sys
import threading
import time

import numpy as np

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

WORKLOADS = {
    # Llama-3.1-8B shape
    "llama8b": dict(model=dict(dim=4096, heads=32, kv=8, layers=32, vocab=128256, ffn=14336, theta=500000.0, eps=1e-5), mode="bfp8",
                    sequences=32, context=2048, name="llama-3.1-8b-shape bfp8, 32 sequences x 2048 context, bf16 KV"),
    # SmolLM-135M shape, batch 1 (the reference's own CPU-runnable case)
    # Mixtral-8x7B shape, attention bfp8, experts bfp4, 64 sequences x 1024 context (one GPU holds it)
    "mixtral": dict(model=dict(dim=4096, heads=32, kv=8, layers=32, vocab=32000, ffn=0, experts=8, k=2, moe=14336, norm_topk=True, theta=1000000.0, eps=1e-5),
                    mode="experts", sequences=64, context=1024, name="mixtral-8x7b-shape, attention bfp8 / experts bfp4, top-2 of 8, 64 sequences x 1024 context, bf16 KV"),
    # Qwen3-30B-A3B shape, bfp8, 128 sessions with contexts drawn uniformly from 256..8192 (seeded)
    "qwen3moe": dict(model=dict(dim=2048, heads=32, kv=4, head_dim=128, layers=48, vocab=151936, ffn=0, experts=128, k=8, moe=768, norm_topk=True, qk_norm=True,
                                theta=1000000.0, eps=1e-6),
                     mode="bfp8", sequences=128, context=8192, ragged=(256, 8192),
                     name="qwen3-30b-a3b-shape bfp8, top-8 of 128, QK-norm, 128 sessions with contexts U{256..8192}, ragged bf16 KV"),
    "smollm": dict(model=dict(dim=576, heads=9, kv=3, layers=30, vocab=49152, ffn=1536, theta=10000.0, eps=1e-5, tied=True), mode="bfp8",
                   sequences=1, context=32, name="smollm-135m-shape bfp8, batch 1, 32-token prompt, bf16 KV"),
}


def parse():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--workload", default="llama8b", choices=sorted(WORKLOADS))
    ap.add_argument("--layers", type=int, default=0, help="fewer blocks than the model has (a smoke run; the JSON line says so)")
    ap.add_argument("--impl", default="ferrite_b200", choices=["ferrite_b200", "reference"])
    ap.add_argument("--reduce", default="peer", choices=["peer", "nccl"], help="several GPUs: how the ranks' partial sums are added")
    ap.add_argument("--parallel", default="tp", choices=["tp", "ep"],
                    help="several GPUs: tp = heads / MLP columns / experts sharded, every rank decodes every sequence, all-reduce after o_proj and "
                         "the MLP; ep (mixtures) = experts AND sequences shared out, whole attention on every rank, tokens to their experts by all-to-all")
    ap.add_argument("--kv", default="bf16", choices=["bf16", "bfp8", "bfp4"], help="the KV cache's format (BASELINE.json's configs keep it in bf16)")
    ap.add_argument("--sweep", type=int, default=1, help="0: leave the isolated matmul sweep out of the line (a profiling run)")
    ap.add_argument("--attend", default="", help="T,H,KV,hd,context[,calls]: only the decode attention, e.g. 32,32,8,128,2048,6")
    ap.add_argument("--matmul", default="", help="M,K,N,fmt[,calls]: only that isolated matmul (RMSNorm + SwiGLU fused), e.g. 32,4096,14336,bfp8,6")
    ap.add_argument("--design", default="", help="binutar[:SIZE], labepel[:SIZE], vunadra[:SIZE] or ronavik[:SIZE]: instead of the workload, prefill and decode of that design at sizes like a real model's layers, "
                                                 "and each of its kernels, beside the Llama decoder at equal size (one GPU)")
    return ap.parse_args()


def measured_peaks():
    try:
        return json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))), "measured"
    except OSError:
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}, "fallback"


class Clocks(threading.Thread):
    """SM clock and throttle reasons sampled through NVML while the timed region runs."""

    def __init__(self, index):
        super().__init__(daemon=True)
        import pynvml
        self.nv, self.samples, self.reasons, self.stop = pynvml, [], set(), False
        pynvml.nvmlInit()
        self.h = pynvml.nvmlDeviceGetHandleByIndex(index)

    def run(self):
        nv = self.nv
        names = {nv.nvmlClocksEventReasonHwSlowdown: "hw_slowdown", nv.nvmlClocksEventReasonHwThermalSlowdown: "hw_thermal_slowdown",
                 nv.nvmlClocksEventReasonSwThermalSlowdown: "sw_thermal_slowdown", nv.nvmlClocksEventReasonSwPowerCap: "sw_power_cap"}
        while not self.stop:
            try:
                self.samples.append(nv.nvmlDeviceGetClockInfo(self.h, nv.NVML_CLOCK_SM))
                mask = nv.nvmlDeviceGetCurrentClocksEventReasons(self.h)
                self.reasons |= {n for bit, n in names.items() if mask & bit}
            except Exception:  # a sample that cannot be read is left out
                pass
            time.sleep(0.05)

    def summary(self):
        self.stop = True
        nv = self.nv
        return {"sm_mhz": float(np.median(self.samples)) if self.samples else None,
                "sm_max_mhz": float(nv.nvmlDeviceGetMaxClockInfo(self.h, nv.NVML_CLOCK_SM)), "reasons": sorted(self.reasons)}


def linear_bytes(c, sequences, fmt_bytes=1.0625, expert_bytes=None):
    """Algorithmic bytes of one step's block-float matmuls: packed weights once, activations in and out (bf16).  A mixture
    reads the experts some token picked: E (1 - (1 - k/E)^T) of them expected (the reference's cost model, ferrite/cost.py:91)."""
    hd = c.head_dim or c.dim // c.heads
    shapes = [(c.dim, (c.heads + 2 * c.kv) * hd, (c.heads + 2 * c.kv) * hd, fmt_bytes), (c.heads * hd, c.dim, c.dim, fmt_bytes)]
    launches = 2
    if getattr(c, "experts", 0):
        tp = getattr(c, "tp", None) or getattr(c, "ep", None)  # expert parallel: a rank reads its share of the touched experts
        everyone = sequences * (tp.world if getattr(c, "ep", None) else 1)  # (c.ep: the other ranks' sequences pick this rank's experts too)
        touched = c.experts * (1 - (1 - c.k / c.experts) ** max(everyone, 1)) / (tp.world if tp else 1)
        eb = expert_bytes or fmt_bytes
        shapes += [(c.dim, c.experts, c.experts, 2.0), (c.dim, touched * 2 * c.moe, touched * c.moe, eb), (touched * c.moe, c.dim, c.dim, eb)]
        launches += 3
    else:
        shapes += [(c.dim, 2 * c.ffn, c.ffn, fmt_bytes), (c.ffn, c.dim, c.dim, fmt_bytes)]
        launches += 2
    per_layer = sum(k * n * b + 2 * sequences * k + 2 * sequences * out for k, n, out, b in shapes)
    head = c.dim * c.vocab_shard * fmt_bytes + 2 * sequences * c.dim + 4 * sequences * c.vocab_shard
    return c.layers * per_layer + head, launches * c.layers + 1


def step_bytes(c, sequences, context_rows, expert_bytes=None, kv_bytes=2.0):
    """Algorithmic bytes a decode step reads per GPU: weights once, the KV rows each token sees (context_rows: their sum
    over the sequences), its embedding row."""
    hd = c.head_dim or c.dim // c.heads
    weights, _ = linear_bytes(c, sequences, expert_bytes=expert_bytes)
    weights -= c.layers * 0  # (activations are part of linear_bytes; they are negligible)
    kv = context_rows * c.layers * 2 * c.kv * hd * kv_bytes
    return weights + kv + sequences * c.dim * 2


def run_ferrite(args):
    import torch
    import torch.distributed as dist
    from ferrite_b200 import llama, ops
    from ferrite_b200.tensor import Runtime, Tensor, jit

    world, rank, local = int(os.environ.get("WORLD_SIZE", 1)), int(os.environ.get("RANK", 0)), int(os.environ.get("LOCAL_RANK", 0))
    assert world == args.gpus, f"--gpus {args.gpus} but WORLD_SIZE is {world}: launch with torch.distributed.run --nproc-per-node {args.gpus}"
    rt = Runtime(local)
    if world > 1:
        dist.init_process_group("nccl", device_id=rt.device)
    wl = WORKLOADS[args.workload]
    full = llama.model(**wl["model"], places=wl["context"] + args.steps + args.warmup + 64)
    if args.layers:
        full.layers = args.layers
    ep = world > 1 and args.parallel == "ep"
    assert not ep or (getattr(full, "experts", 0) and wl["sequences"] % world == 0), "--parallel ep: a mixture, its sequences shared out evenly"
    c = llama.expert_parallel(full, rank, world, dist.group.WORLD) if ep else llama.tensor_parallel(full, rank, world, dist.group.WORLD) if world > 1 else full
    if world == 1:
        c.vocab_shard = full.vocab
    reduction = "none"
    if ep:
        reduction = "none (two all-to-alls a block: tokens to their experts' ranks and back)"
    elif world > 1:
        reduction = "nccl all-reduce + add"
        if args.reduce == "peer":
            why = ""
            try:  # this library's kernel over NVLink peer memory; NCCL's all-reduce if the mapping cannot be set up here
                llama.peer_reduce(rt, c, wl["sequences"])
            except Exception as e:  # noqa: BLE001
                why = type(e).__name__
            ok = torch.tensor([0 if why else 1], device=rt.device)
            dist.all_reduce(ok, op=dist.ReduceOp.MIN)  # every rank takes the same path
            if int(ok.item()):
                reduction = "fb_peer_reduce_add (own kernel, peer loads over NVLink, residual fused)"
            else:
                c.tp.peer = None
                reduction += f" (peer memory unavailable on some rank{': ' + why if why else ''})"
    prec = llama.precision(full, wl["mode"])
    w = llama.random_weights(rt, c, prec, seed=0, full=full)
    S_all, ctx = wl["sequences"], wl["context"]
    S = S_all // world if ep else S_all  # the sequences this rank decodes
    part = ctx + args.steps + args.warmup + 64
    part += -part % 64
    rng = np.random.default_rng(0)
    # where each sequence stands: all at `context`, or (a serving mix) contexts drawn uniformly, seeded
    ctxs = [int(v) for v in rng.integers(wl["ragged"][0], wl["ragged"][1] + 1, S_all)] if wl.get("ragged") else [ctx] * S_all
    ctxs = ctxs[rank * S:(rank + 1) * S] if ep else ctxs
    moe = bool(getattr(full, "experts", 0))
    expert_bytes = 0.5625 if wl["mode"] == "experts" else None
    hd = llama.head(full)
    caches = []
    gen = torch.Generator(device=rt.device).manual_seed(1 + rank)
    for _ in range(full.layers):  # the prompts' keys and values: N(0, 1), as a prefill would have left them
        t = Tensor(rt, S * part, hd, batch=2 * c.kv)
        t.buf.normal_(0, 1, generator=gen)
        caches.append(t if args.kv == "bf16" else t.cast(args.kv).realize())  # (a block-float cache: rounded as a put rounds)
    kv_bytes = {"bf16": 2.0, "bfp8": 1.0625, "bfp4": 0.5625}[args.kv]
    slots = S if S > 1 else None

    def step_fn(ids, places):
        return llama.next_tokens(llama.forward(ids, places, w, c, caches, slots), c)

    step = jit(step_fn)
    on = lambda row: Tensor.of(rt, [row], "int32")
    ids0 = [int(v) for v in rng.integers(0, full.vocab, S_all)]
    ids0 = ids0[rank * S:(rank + 1) * S] if ep else ids0
    place = 0  # steps taken so far: sequence u stands at ctxs[u] + place
    at = lambda: [v + place for v in ctxs]
    # the first two calls plan and record; they are part of the warm-up
    before = ops.KERNELS[0]
    picks = step(on(ids0), on(at()))
    place += 1
    per_step = None
    for i in range(max(args.warmup, 3) - 1):
        k0 = ops.KERNELS[0]
        picks = step(on(picks.numpy().reshape(-1).tolist()), on(at()))
        if i == 0:
            per_step = ops.KERNELS[0] - k0  # kernels the recorded step holds (counted while it was recorded)
        place += 1
    rt.wait()

    # ---- device-resident loop: the pick feeds the next step on the device, places advance on the device
    ids_t, places_t = on(picks.numpy().reshape(-1).tolist()), on(at())
    one = Tensor.of(rt, [[1] * S], "int32")
    bump = jit(lambda p: p + one)  # (records on its second call)

    def sync_all():
        torch.cuda.synchronize()
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    for _ in range(3):
        places_t = bump(places_t)
    clocks = Clocks(local)
    clocks.start()
    sync_all()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(args.steps):
        out = step(ids_t, places_t)
        ids_t.buf.copy_(out.buf, non_blocking=True)
        places_t = bump(places_t)
    e1.record()
    sync_all()
    ms = e0.elapsed_time(e1)
    place += args.steps + 3

    # ---- end to end: host ids and places in (pinned), picked tokens out, every step
    h_ids = torch.tensor([ids0], dtype=torch.int32).pin_memory()
    h_places = torch.tensor([at()], dtype=torch.int32).pin_memory()
    h_out = torch.empty(1, 1, S, dtype=torch.int32).pin_memory()
    d_ids, d_places = on(ids0), on(at())
    e2e_steps = max(8, args.steps // 2)
    sync_all()
    e2, e3 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e2.record()
    for _ in range(e2e_steps):
        d_ids.buf.copy_(h_ids.view(1, 1, S), non_blocking=True)
        d_places.buf.copy_(h_places.view(1, 1, S), non_blocking=True)
        out = step(d_ids, d_places)
        h_out.copy_(out.buf, non_blocking=True)
        torch.cuda.current_stream().synchronize()
        h_ids.copy_(h_out.view(1, S))  # the next step's input is this step's pick, from the host
        h_places += 1
    e3.record()
    sync_all()
    ms_e2e = e2.elapsed_time(e3)
    clk = clocks.summary()
    if getattr(getattr(c, "tp", None), "peer", None) is not None:
        c.tp.peer.check()

    mm = None
    lin_bytes, lin_launches = linear_bytes(c, S, expert_bytes=expert_bytes)
    lin_ms = 0.0
    # ---- the dominant kernel alone: the step's block-float matmuls, back to back, every weight of the model once
    # (a dense model; a mixture's indexed matmuls depend on the router's picks, so its roofline is the whole step's)
    if not moe:
        x32 = Tensor.of(rt, rng.normal(0, 1, (S, full.dim)).astype(np.float32).tolist())
        f32 = Tensor.of(rt, rng.normal(0, 1, (S, c.ffn)).astype(np.float32).tolist())
        a32 = Tensor.of(rt, rng.normal(0, 1, (S, c.heads * hd)).astype(np.float32).tolist())

        def matmuls():
            for p in w["_blocks"]:
                x32.matmul(p["qkv_proj"]).realize()
                a32.matmul(p["o_proj"]).realize()
                x32.matmul(p["gate_up_proj"]).realize()
                f32.matmul(p["down_proj"]).realize()
            return x32.matmul(w["embed.T"], dtype="fp32").realize()

        mm = jit(lambda: matmuls())
        for _ in range(3):
            mm()
        torch.cuda.synchronize()
        e4, e5 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        reps = 5
        e4.record()
        for _ in range(reps):
            mm()
        e5.record()
        torch.cuda.synchronize()
        lin_ms = e4.elapsed_time(e5) / reps

    # ---- time to first token (one GPU, a dense model): one sequence's prompt of `context` tokens from place 0 in chunks of
    # 128 through the same kernels (the matmuls at 128 rows a pass, the prefill-shaped attention), then the greedy pick
    # (the reference's B3, test/benchmark.py:172-181, times the same call on its side)
    ttft = None
    if world == 1 and not moe:
        prompt = [int(v) for v in rng.integers(0, full.vocab, ctx)]
        one = llama.kv_cache(c, part, llama.zeros(rt))
        tries = []
        for _ in range(2):  # (the first pass also plans and allocates)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            first = llama.next_tokens(llama.prefill(prompt, w, c, one, 128, on), c).numpy()
            tries.append(time.perf_counter() - t0)
        ttft = {"ms": 1e3 * tries[-1], "prompt_tokens": ctx, "chunk": 128, "tokens_per_s": ctx / tries[-1],
                "what": "one sequence's prompt from place 0 to its first token on the host, wall clock, second of two passes"}
        del one

    # max over ranks
    times = torch.tensor([ms, ms_e2e, lin_ms], device=rt.device)
    if world > 1:
        dist.all_reduce(times, op=dist.ReduceOp.MAX)
    ms, ms_e2e, lin_ms = times.tolist()
    peaks, peak_kind = measured_peaks()
    rows_seen = sum(ctxs) + S * (args.warmup + args.steps // 2)  # KV rows the middle step of the timed run reads
    whole = step_bytes(c, S, rows_seen, expert_bytes, kv_bytes)
    if moe:  # the roofline of a mixture's step as a whole: every kernel of it streams weights or KV rows
        lin_bytes, lin_launches, lin_ms = whole, int(per_step or 1), ms / args.steps
    achieved = lin_bytes / (lin_ms * 1e-3) / 1e9
    line = {
        "metric": "decode tokens/s", "value": S_all * args.steps / (ms * 1e-3), "unit": "tokens/s", "n_gpus": world, "steps": args.steps,
        "warmup": max(args.warmup, 3), "ms_per_step": ms / args.steps, "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic",
        "config": {"workload": wl["name"], "layers": full.layers, "parallelism": (f"dp{world} (sequences, whole attention) + ep{world} (experts), all-to-all dispatch and return" if ep else
                                                                             f"tp{world}" + (f" (attention heads) + ep{world} (experts), all-reduce after o_proj and after the experts" if moe and world > 1 else "")), "reduction": reduction, "l2": "inputs larger than L2 (every step streams all weights and KV rows)",
                   "weights": "random N(0, 0.02) quantised on the device", "kv": "N(0, 1) %s standing in for the prompts' prefill" % args.kv},
        "e2e": {"value": S_all * e2e_steps / (ms_e2e * 1e-3), "unit": "tokens/s", "h2d_bytes_per_step": 2 * 4 * S_all, "d2h_bytes_per_step": 4 * S_all, "steps": e2e_steps},
        "gpu_launches": int(per_step or 0) * args.steps,
        "clocks": clk,
        "roofline": {"bound": "hbm", "kernel": ("the whole decode step (indexed block-float matmuls + decode attention), %d tokens" if moe else
                                                "linear_tcgen05_kernel / linear_persistent_kernel (block-float dequant GEMM: a CTA per tile, or persistent with at least a tile per SM; %d tokens)") % S, "achieved": achieved,
                     "peak": peaks["hbm_gbs"], "unit": "GB/s", "frac": achieved / peaks["hbm_gbs"], "peak_source": peak_kind,
                     "traffic": None if moe else 1.002 * lin_bytes / lin_launches,
                     "traffic_source": "not captured for the whole step" if moe else "algorithmic bytes x 1.002 (DRAM read+write of the ncu capture in profiles/, 4096x14336 bfp8, 32 tokens)",
                     "launches": lin_launches, "us_per_launch": lin_ms * 1e3 / lin_launches, "bytes_per_launch": lin_bytes / lin_launches},
        "step_roofline": {"algorithmic_bytes_per_gpu": whole, "frac_of_hbm": whole / (ms / args.steps * 1e-3) / 1e9 / peaks["hbm_gbs"]},
    }
    if ttft:
        line["ttft"] = ttft
    if rank == 0 and world == 1:
        del w, caches, step, mm
        torch.cuda.empty_cache()
        if args.sweep and not moe:
            line["matmul_sweep"] = matmul_sweep(rt.device, peaks["hbm_gbs"])
        line["cpu_baseline"] = cpu_baseline(args, sample_seconds=20)
    if rank == 0:
        print(json.dumps(line), flush=True)
    if world > 1:  # leave without tearing NCCL down: the recorded graphs still hold its kernels, and a teardown waits on them
        dist.barrier()
        torch.cuda.synchronize()
        sys.stdout.flush()
        os._exit(0)


def one_matmul(spec):
    """--matmul: a few eager calls of one isolated matmul over four weight copies (what an ncu capture of the kernel runs)."""
    import torch
    from ferrite_b200 import ops
    parts = spec.split(",")
    M, K, N, fmt, calls = int(parts[0]), int(parts[1]), int(parts[2]), parts[3], int(parts[4]) if len(parts) > 4 else 6
    device, gen = torch.device("cuda:0"), torch.Generator(device="cuda:0").manual_seed(0)
    g = (1 + 0.1 * torch.randn(K, device=device, generator=gen)).bfloat16()
    ws = [ops.quantize((torch.randn(K, N, device=device, generator=gen) * 0.02).bfloat16(), fmt) for _ in range(4)]
    x = torch.randn(M, K, device=device, generator=gen).bfloat16()
    out = torch.empty(M, N // 2, device=device, dtype=torch.bfloat16)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(calls):
        ops.linear(x, ws[i % 4], out=out, norm_w=g, eps=1e-5, epilogue="swiglu")
    e1.record()
    torch.cuda.synchronize()
    print(json.dumps({"matmul": spec, "calls": calls, "us_per_call_eager": e0.elapsed_time(e1) * 1e3 / calls}))


def one_attention(spec):
    """--attend: a few eager calls of the decode attention alone, every sequence at the same context, each call over its
    own KV cache (four of them, together larger than L2): what an ncu capture of the kernel runs."""
    import torch
    from ferrite_b200 import ops
    parts = [int(v) for v in spec.split(",")]
    T, H, KV, hd, ctx, calls = parts[:5] + [parts[5] if len(parts) > 5 else 6]
    device, gen = torch.device("cuda:0"), torch.Generator(device="cuda:0").manual_seed(0)
    part = ctx + 64 - ctx % 64
    caches = [torch.empty(2 * KV, T * part, hd, device=device, dtype=torch.bfloat16).normal_(0, 1, generator=gen) for _ in range(4)]
    q = torch.randn(T, H * hd, device=device, generator=gen).bfloat16()
    base = torch.arange(T, device=device, dtype=torch.int32) * part
    place = torch.full((T,), ctx - 1, device=device, dtype=torch.int32)
    out = torch.empty(T, H * hd, device=device, dtype=torch.bfloat16)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(calls):
        ops.decode_attention(q, caches[i % 4], base, place, H, KV, hd, ctx, out=out)
    e1.record()
    torch.cuda.synchronize()
    kv_bytes = T * ctx * 2 * KV * hd * 2
    print(json.dumps({"attend": spec, "calls": calls, "us_per_call_eager": e0.elapsed_time(e1) * 1e3 / calls, "kv_bytes_per_call": kv_bytes}))


# layers of the sizes real models have, latent and linear mixers in turn, a Llama-like decoder of the same width, depth and MLP
# beside each (its attention at that width's usual head counts)
DESIGN_SIZES = {
    "4096": dict(width=4096, layers=8, ff=14336, vocab=32000, heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536, kv=8),
    "2560": dict(width=2560, layers=8, ff=6400, vocab=32000, heads=32, dim=64, rot_dim=32, vdim=64, kv_rank=256, q_rank=768, kv=8),
}

# grouped-query attention within spans and a mixture of experts with a shared one, at a Mixtral-like and a Qwen3-30B-A3B-like size, a
# Llama-like mixture of the same heads, experts and depth beside each
LABEPEL_SIZES = {
    "4096": dict(width=4096, layers=6, vocab=32000, heads=32, kv=8, dim=128, vdim=128, span=8192, experts=8, top=2, ff=14336, shared=14336),
    "2048": dict(width=2048, layers=8, vocab=32000, heads=32, kv=4, dim=128, vdim=128, span=8192, experts=128, top=8, ff=768, shared=768),
}


# a layer of each kind - attention with a short convolution before a dense feed-forward, attention whose values are its keys and
# attention over latents, both within a window, before a mixture - run twice in a loop; a Llama-like mixture of the same heads,
# experts and layer runs beside it
VUNADRA_SIZES = {
    "4096": dict(width=4096, layers=6, vocab=32000, heads=32, kv=8, dim=128, vdim=128, conv=4, window=1024, rot_dim=64, kv_rank=512, experts=8, identity=1, top=2, ff=14336, dense=14336),
    "2048": dict(width=2048, layers=6, vocab=32000, heads=32, kv=4, dim=128, vdim=128, conv=4, window=1024, rot_dim=64, kv_rank=512, experts=128, identity=8, top=8, ff=768, dense=6144),
}


# state spaces of Mamba-2's usual shape and attention beside a gated recurrence in turn, each before a mixture; a Llama-like mixture of the
# same heads, experts and depth beside it
RONAVIK_SIZES = {
    "4096": dict(width=4096, layers=6, vocab=32000, heads=32, kv=8, dim=128, vdim=128, lru=4096, blocks=32, conv=4, ssm_heads=128, ssm_vdim=64, state=128, groups=8, experts=8, top=2, ff=14336),
    "2048": dict(width=2048, layers=8, vocab=32000, heads=32, kv=4, dim=128, vdim=128, lru=2048, blocks=16, conv=4, ssm_heads=64, ssm_vdim=64, state=128, groups=8, experts=128, top=8, ff=768),
}


def ronavik_models(s, places):
    """(Ronavik config, Llama config of a mixture) of one size."""
    from ferrite_b200 import llama, ronavik
    mlp = dict(kind="moe", router=dict(experts=s["experts"], top=s["top"]), expert=dict(ff=s["ff"]))
    space = dict(type="mamba2", mixer=dict(heads=s["ssm_heads"], vdim=s["ssm_vdim"], state=s["state"], groups=s["groups"], conv=s["conv"], norm_groups=s["groups"]), mlp=mlp)
    left = dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["vdim"], scale=s["dim"] ** -0.5, q_temp=dict(coef=0.1, every=8192))
    side = dict(type="parallel", mixer=dict(left=left, right=dict(width=s["lru"], blocks=s["blocks"], conv=s["conv"]), left_scale=1.0, right_scale=1.0), mlp=mlp)
    return (ronavik.model(vocab=s["vocab"], dim=s["width"], eps=1e-5, blocks=[space, side] * (s["layers"] // 2), positions=places, places=places),
            llama.model(dim=s["width"], heads=s["heads"], kv=s["kv"], head_dim=s["dim"], layers=s["layers"], vocab=s["vocab"], ffn=0, experts=s["experts"], k=s["top"], moe=s["ff"], theta=10000.0,
                        eps=1e-5, places=places))


def vunadra_models(s, places):
    """(Vunadra config, Llama config of a mixture) of one size."""
    from ferrite_b200 import llama, vunadra
    heads, d = dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["vdim"], scale=s["dim"] ** -0.5), s["dim"]
    mixture = dict(kind="moe", router=dict(experts=s["experts"], identity=s["identity"], top=s["top"], scale=1.0), expert=dict(ff=s["ff"], limit=7.0))
    yarn, waves = dict(factor=4.0, original=4096, fast=32.0, slow=1.0), dict(factor=8.0, low=1.0, high=4.0, original=8192)
    blocks = [dict(type="attention", mixer=heads | dict(conv=s["conv"], rot=dict(base=500000.0, dims=d, scaling=yarn)), mlp=dict(kind="dense", ff=s["dense"])),
              dict(type="attention_2", mixer=heads | dict(mask=dict(size=s["window"]), softcap=30.0, rot=dict(base=500000.0, dims=d, scaling=waves)), mlp=mixture),
              dict(type="latent_attention", mixer=dict(heads=s["heads"], dim=d, rot_dim=s["rot_dim"], vdim=s["vdim"], kv_rank=s["kv_rank"], mask=dict(size=s["window"]), scale=(d + s["rot_dim"]) ** -0.5,
                                                       rot=dict(base=500000.0, dims=s["rot_dim"])), mlp=mixture)]
    return (vunadra.model(vocab=s["vocab"], dim=s["width"], eps=1e-5, blocks=blocks, loop=dict(start=0, stop=3, times=s["layers"] // 3), places=places),
            llama.model(dim=s["width"], heads=s["heads"], kv=s["kv"], head_dim=d, layers=s["layers"], vocab=s["vocab"], ffn=0, experts=s["experts"], k=s["top"], moe=s["ff"], theta=10000.0,
                        eps=1e-5, places=places))


def labepel_models(s, places):
    """(Labepel config, Llama config of a mixture) of one size."""
    from ferrite_b200 import labepel, llama
    block = dict(type="attention", mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["vdim"], mask=dict(size=s["span"]), scale=s["dim"] ** -0.5, v_mix=True),
                 mlp=dict(kind="moe", router=dict(experts=s["experts"], top=s["top"]), expert=dict(ff=s["ff"]), shared=dict(ff=s["shared"])))
    return (labepel.model(vocab=s["vocab"], dim=s["width"], eps=1e-5, blocks=[block] * s["layers"], positions=places, places=places),
            llama.model(dim=s["width"], heads=s["heads"], kv=s["kv"], head_dim=s["dim"], layers=s["layers"], vocab=s["vocab"], ffn=0, experts=s["experts"], k=s["top"], moe=s["ff"], theta=10000.0,
                        eps=1e-5, places=places))


def design_models(s, places):
    """(Binutar config, Llama config) of one size."""
    from ferrite_b200 import binutar, llama
    rot = dict(base=10000.0, dims=s["rot_dim"], scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))
    latent = dict(heads=s["heads"], dim=s["dim"], rot_dim=s["rot_dim"], vdim=s["vdim"], kv_rank=s["kv_rank"], q_rank=s["q_rank"], rot=rot, scale=(s["dim"] + s["rot_dim"]) ** -0.5)
    linear = dict(heads=s["heads"], dim=s["dim"], vdim=s["vdim"], decay=[1 - 2.0 ** -(2 + 6 * h / s["heads"]) for h in range(s["heads"])])
    mlp = dict(kind="dense", ff=s["ff"], limit=7.0)
    blocks = [dict(type="lightning", mixer=linear, mlp=mlp) if i % 2 else dict(type="latent_attention", mixer=latent, mlp=mlp) for i in range(s["layers"])]
    return (binutar.model(vocab=s["vocab"], dim=s["width"], eps=1e-5, blocks=blocks, places=places),
            llama.model(dim=s["width"], heads=s["heads"], kv=s["kv"], head_dim=128 if s["dim"] == 128 else 64, layers=s["layers"], vocab=s["vocab"], ffn=s["ff"], theta=10000.0,
                        eps=1e-5, places=places))


def timed(calls, copies, call):
    """Microseconds of call(i), i running round `copies` sets of inputs, from a replayed graph of `calls` of them."""
    import torch
    for i in range(3):
        call(i % copies)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(calls):
            call(i % copies)
    best = 1e30
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        graph.replay()
        e1.record()
        torch.cuda.synchronize()
        best = min(best, e0.elapsed_time(e1) * 1e3 / calls)
    return best


def design_steps(rt, c, prec, S, ctx, prompt, steps):
    """Decode of S sequences at ctx tokens each (a recorded step of distinct tokens) and one sequence's prompt."""
    import torch
    from ferrite_b200 import llama, models
    from ferrite_b200.tensor import Tensor, jit
    family = models.of(c)
    w = family.random_weights(rt, c, prec)
    part = ctx + 64 + steps
    part += -part % 64
    kv = family.kv_cache(c, S * part, llama.zeros(rt), S)
    gen = torch.Generator(device=rt.device).manual_seed(1)
    for t in [t for x in kv for t in (x if isinstance(x, tuple) else (x,)) if t is not None]:  # (what the prompts would have left)
        t.buf.normal_(0, 1, generator=gen)
    on = lambda row: Tensor.of(rt, [row], "int32")
    step = jit(lambda ids, at: llama.next_tokens(family.forward(ids, at, w, c, kv, S), c))
    ids, one = on([(37 * i + 1) % c.vocab for i in range(S)]), Tensor.of(rt, [[1] * S], "int32")  # (the same every step: a mixture's sequences would else fall into step)
    bump = jit(lambda p: p + one)
    at = on([ctx] * S)
    before = rt.launches
    for i in range(4):
        out = step(ids, at)
        at = bump(at)
        if i == 0:
            names = rt.profile(before)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps):
        out = step(ids, at)
        at = bump(at)
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    rows = {"decode": {"sequences": S, "context": ctx, "ms_per_step": ms, "tokens/s": 1e3 * S / ms, "launches": dict(names)}, "prefill": []}
    alone = family.kv_cache(c, prompt + 64, llama.zeros(rt), 1)
    tokens = [int(v) for v in np.random.default_rng(0).integers(0, c.vocab, prompt)]
    for chunk in (prompt, 512, 128):
        tries = []
        for _ in range(3):
            torch.cuda.synchronize()
            e0.record()
            llama.next_tokens(llama.prefill(tokens, w, c, alone, chunk, on), c)
            e1.record()
            torch.cuda.synchronize()
            tries.append(e0.elapsed_time(e1))
        rows["prefill"].append({"prompt": prompt, "chunk": chunk, "ms": min(tries), "tokens/s": 1e3 * prompt / min(tries)})
    rt.wait()
    return rows


def design_kernels(rt, s, T, ctx, peaks):
    """Each kernel of a layer at T tokens - a decode step of T sequences, or (ctx 0) a prompt of T tokens - alone, over inputs that
    together exceed L2, with the part of its roofline that it reaches: bytes by the measured copy bandwidth or products by the
    measured bf16 rate, whichever takes longer.  Then the Llama decoder's like kernels."""
    import torch
    from ferrite_b200 import _lib, ops
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen).bfloat16()
    f32 = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen)
    rows, prompt = [], ctx == 0
    d, H, dim, rd, vd, rank, qr, ff = (s[k] for k in ("width", "heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "ff"))

    def row(name, us, nbytes, flops=0.0, like=None):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)} | ({"like": like} if like else {}))

    def dense(name, K, N, batch=1, kind=_lib.DENSE_NONE, out_dtype=torch.bfloat16, like="fb_linear"):
        copies = max(1, min(16, int(3e8 // (2 * batch * K * N))))
        ws = [bf(batch, N, K) for _ in range(copies)]
        x = bf(T, batch, K).permute(1, 0, 2)
        cols = N // 2 if kind == _lib.DENSE_GLU else N
        out = torch.empty(T, batch, cols, device=dev, dtype=out_dtype).permute(1, 0, 2)
        v, extra, more = f32(N), {}, 0
        if kind == _lib.DENSE_SILU:
            extra = dict(act_cols=N // 2)
        if kind == _lib.DENSE_GLU:
            extra = dict(limit=7.0, slope=1.702)
        if kind == _lib.DENSE_GATE:
            g = f32(T, batch)
            extra = dict(gate=g.data_ptr(), ld_gate=batch)
        if kind == _lib.DENSE_DYT_ADD:
            res, h = f32(T, N), bf(T, N)
            extra = dict(residual=res.data_ptr(), ld_residual=N, alpha=v.data_ptr(), w=v.data_ptr(), b=v.data_ptr(), h_out=h.data_ptr(), ld_h=N, alpha2=v.data_ptr(),
                         w2=v.data_ptr(), b2=v.data_ptr())
            more = 6 * T * N
        us = timed(40, copies, lambda i: ops.dense(x, ws[i].transpose(1, 2), out, True, kind, **extra))
        row(f"fb_dense {name} {batch}x[{K}, {N}]" if batch > 1 else f"fb_dense {name} [{K}, {N}]", us,
            2 * batch * K * N + 2 * T * batch * K + out.element_size() * T * batch * cols + more, 2.0 * T * batch * K * N, like)

    dense("in", d, qr + rank + rd + H, out_dtype=torch.float32)
    dense("uq", qr, H * (dim + rd))
    dense("uk by head", dim, rank, H)
    dense("uv by head, gate", rank, vd, H, _lib.DENSE_GATE)
    dense("o, dyt, add, dyt", H * vd, d, 1, _lib.DENSE_DYT_ADD, torch.float32)
    dense("qkvg, silu", d, 2 * H * (dim + vd), 1, _lib.DENSE_SILU)
    dense("gate_up, clamped unit", d, 2 * ff, 1, _lib.DENSE_GLU)
    dense("down, dyt, add, dyt", ff, d, 1, _lib.DENSE_DYT_ADD, torch.float32)
    dense("head", d, s["vocab"], out_dtype=torch.float32)

    W, keys = rank + rd, T if prompt else ctx
    part = keys + -keys % 64
    caches = [bf((1 if prompt else T) * part, W) for _ in range(4)]
    q, o, sink = bf(T, H * W), torch.empty(T, H * rank, device=dev, dtype=torch.bfloat16), f32(H)
    base = torch.arange(T, device=dev, dtype=torch.int32) * part
    last = torch.arange(T, device=dev, dtype=torch.int32) if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    pairs = T * (T + 1) / 2 if prompt else T * ctx
    us = timed(20, 4, lambda i: ops.latent_attention(q, caches[i], None if prompt else base, last, H, rank, 0.1, sink, keys, prompt, out=o))
    row("fb_latent_attention", us, 2 * ((1 if prompt else T) * keys * W + T * H * (W + rank)), 2.0 * pairs * H * (W + rank), "attention")
    if prompt:  # (the same attention with keys and values made first: fewer products, and what a kernel of that form would be held to)
        row("fb_latent_attention, counted as keys and values of a head", us, 0, 2.0 * pairs * H * (dim + rd + vd), "attention")

    down, places = f32(T, qr + W + H), last if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    at, freq, cq = (places if prompt else base + places), torch.ones(rd // 2, device=dev, dtype=torch.float64), bf(T, qr)
    us = timed(40, 1, lambda i: ops.latent_put(down, qr, rank, rd, rd, f32_ones(dev, qr), f32_ones(dev, rank), 1e-5, freq, 1.0, places, at, caches[0], cq))
    row("fb_latent_put", us, T * (qr + W) * 6, like="fb_rope_kv_write")
    qh, q3 = bf(T, H, dim + rd), q.view(T, H, W).permute(1, 0, 2)
    us = timed(40, 1, lambda i: ops.rotate_pairs(qh.permute(1, 0, 2)[:, :, dim:], (freq, rd, 1.0), places, q3[:, :, rank:]))
    row("fb_rotate_pairs", us, 4 * T * H * rd, like="fb_rope_kv_write")

    n = 2 * H * (dim + vd)
    qkvg, out, decay = bf(T, n), f32(T, H * vd), torch.full((H,), 0.95, device=dev)
    states = [f32(1 if prompt else T, H * dim, vd) for _ in range(1 if prompt else 4)]
    us = timed(20, len(states), lambda i: ops.decay_scan(qkvg, H, dim, vd, decay, places, -1 if prompt else keys + 9, states[i], out))
    row("fb_decay_scan", us, T * H * (2 * (2 * dim + vd) + 4 * vd) + (1 if prompt else T) * H * dim * vd * 8, 2.0 * T * H * 2 * dim * vd)
    g, h = qkvg[:, n - H * vd:], bf(T, H * vd)
    us = timed(40, 1, lambda i: ops.gated_rmsnorm(out, g, f32_ones(dev, H * vd), 1e-5, h))
    row("fb_gated_rmsnorm", us, T * H * vd * 8, like="fb_rmsnorm")
    return rows


_ONES = {}


def f32_ones(dev, n):
    import torch
    if (dev, n) not in _ONES:
        _ONES[dev, n] = torch.ones(n, device=dev)
    return _ONES[dev, n]


def llama_kernels(rt, s, T, ctx, peaks):
    """The Llama decoder's kernels at the same size (bfp8 weights, as it serves them), likewise."""
    import torch
    from ferrite_b200 import ops
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen).bfloat16()
    rows, prompt = [], ctx == 0
    d, H, KV, ff, hd = s["width"], s["heads"], s["kv"], s["ff"], 128 if s["dim"] == 128 else 64

    def row(name, us, nbytes, flops=0.0):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)})

    for name, K, N, epilogue, norm in (("qkv, rms", d, (H + 2 * KV) * hd, "none", True), ("o, add", H * hd, d, "residual", False), ("gate_up, rms, swiglu", d, 2 * ff, "swiglu", True),
                                       ("down, add", ff, d, "residual", False), ("head, rms", d, s["vocab"], "none", True)):
        copies = max(1, min(16, int(3e8 // (1.0625 * K * N))))
        ws = [ops.quantize(bf(K, N), "bfp8") for _ in range(copies)]
        x, g, res = bf(T, K), bf(K), bf(T, N)
        cols = N // 2 if epilogue == "swiglu" else N
        out = torch.empty(T, cols, device=dev, dtype=torch.bfloat16)
        us = timed(40 if not prompt else 8, copies, lambda i: ops.linear(x, ws[i], out=out, norm_w=g if norm else None, epilogue=epilogue, residual=res if epilogue == "residual" else None))
        row(f"fb_linear bfp8 {name} [{K}, {N}]", us, 1.0625 * K * N + 2 * T * K + 2 * T * cols + (2 * T * N if epilogue == "residual" else 0), 2.0 * T * K * N)
    keys = T if prompt else ctx
    part = keys + -keys % 64
    caches = [bf(2 * KV, (1 if prompt else T) * part, hd) for _ in range(4)]
    q, o = bf(T, H * hd), torch.empty(T, H * hd, device=dev, dtype=torch.bfloat16)
    base = torch.arange(T, device=dev, dtype=torch.int32) * part
    last = torch.arange(T, device=dev, dtype=torch.int32) if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    pairs = T * (T + 1) / 2 if prompt else T * ctx
    if prompt:
        us = timed(8, 4, lambda i: ops.prefill_attention(q, caches[i], 0, last, H, KV, hd, keys, out=o))
    else:
        us = timed(20, 4, lambda i: ops.decode_attention(q, caches[i], base, last, H, KV, hd, keys, out=o))
    row("fb_prefill_attention" if prompt else "fb_decode_attention", us, 2 * ((1 if prompt else T) * keys * 2 * KV * hd + 2 * T * H * hd), 4.0 * pairs * H * hd)
    qkv, cos = bf(T, (H + 2 * KV) * hd), bf(keys + 1, hd)
    at = last if prompt else base + last
    us = timed(40, 1, lambda i: ops.rope_kv_write(qkv, cos, cos, last, at, caches[0], H, KV, hd, q_out=q))
    row("fb_rope_kv_write", us, 4 * T * (H + 2 * KV) * hd)
    x, g = bf(T, d), bf(d)
    us = timed(40, 1, lambda i: ops.rmsnorm(x, g, 1e-5, out=o[:, :d] if H * hd >= d else None))
    row("fb_rmsnorm", us, 4 * T * d)
    return rows


def labepel_kernels(rt, s, T, ctx, peaks):
    """Each kernel of a Labepel layer, as design_kernels does it."""
    import torch
    from ferrite_b200 import _lib, ops
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    f32 = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen)
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.bfloat16).normal_(0, 1, generator=gen)
    rows, prompt = [], ctx == 0
    d, H, G, dim, vd, E, k, ff, sff = (s[n] for n in ("width", "heads", "kv", "dim", "vdim", "experts", "top", "ff", "shared"))

    def row(name, us, nbytes, flops=0.0, like=None):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)} | ({"like": like} if like else {}))

    def dense(name, K, N, kind=_lib.DENSE_NONE, out_dtype=torch.bfloat16, like="fb_linear"):
        copies = max(1, min(16, int(3e8 // (2 * K * N))))
        ws, x, cols = [bf(1, N, K) for _ in range(copies)], bf(1, T, K), N // 2 if kind == _lib.DENSE_SWIGLU else N
        out = torch.empty(1, T, cols, device=dev, dtype=out_dtype)
        us = timed(40, copies, lambda i: ops.dense(x, ws[i].transpose(1, 2), out, True, kind))
        row(f"fb_dense {name} [{K}, {N}]", us, 2 * K * N + 2 * T * K + out.element_size() * T * cols, 2.0 * T * K * N, like)

    n = (H + G) * dim + G * vd
    dense("in", d, n + H * vd + E, out_dtype=torch.float32)
    dense("o", H * vd, d)
    dense("shared gate_up, swiglu", d, 2 * sff, _lib.DENSE_SWIGLU)
    dense("shared down", sff, d)
    dense("head", d, s["vocab"], out_dtype=torch.float32)

    joint, keys = f32(T, n + H * vd + E), T if prompt else ctx
    part = keys + -keys % 64
    caches = [bf(G, (1 if prompt else T) * part, dim + vd) for _ in range(4)]
    last = torch.arange(T, device=dev, dtype=torch.int32) if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    base = torch.arange(T, device=dev, dtype=torch.int32) * part
    at, q, o = (last if prompt else base + last), bf(T, H * dim), bf(T, H * vd)
    us = timed(40, 1, lambda i: ops.heads_put(joint, H, G, dim, vd, at, caches[0], q, f32_ones(dev, n), f32_ones(dev, dim), f32_ones(dev, dim), 1e-5, joint[:, n:n + G * vd], f32_ones(dev, G * vd),
                                              f32_ones(dev, 1)))
    row("fb_heads_put", us, T * (4 * (n + G * vd) + 2 * n), like="fb_rope_kv_write")
    sink, gate, pairs = f32(H), joint[:, n:n + H * vd], T * (T + 1) / 2 if prompt else T * ctx
    us = timed(20, 4, lambda i: ops.heads_attention(q, caches[i], None if prompt else base, last, H, vd, 0.1, keys, prompt, s["span"], sink, gate, out=o))
    row("fb_heads_attention", us, 2 * ((1 if prompt else T) * keys * G * (dim + vd) + T * H * (dim + vd)) + 4 * T * H * vd, 2.0 * pairs * H * (dim + vd), "attention")

    logits = f32(T, E)
    us = timed(40, 1, lambda i: ops.route(logits, E, k, f32_ones(dev, E)))
    row("fb_route", us, T * (4 * E + 12 * k), like="fb_topk and fb_touched (fb_group)")
    r = ops.route(logits, E, k)
    touched, live = len(set(r.ids.cpu().reshape(-1).tolist())), int(r.live)
    copies = max(1, min(4, int(3e8 // (6 * touched * d * ff)) + 1))
    gate_up, down, h = [bf(E, 2 * ff, d).transpose(1, 2) for _ in range(copies)], [bf(E, d, ff).transpose(1, 2) for _ in range(copies)], bf(T, d)
    x, act, y = bf(r.tiles * r.tile, d), bf(r.tiles * r.tile, ff), bf(r.tiles * r.tile, d)
    if not r.shared:
        us = timed(20, 1, lambda i: ops.spread_rows(h, r, x))
        row("fb_spread_rows", us, 2 * T * (k + 1) * d, like="fb_gather_rows")
    us = timed(20, copies, lambda i: ops.grouped(h if r.shared else x, gate_up[i], r, act, _lib.DENSE_SWIGLU, r.shared))
    row(f"fb_dense_grouped gate_up, swiglu ({touched} experts, {live} tiles of {r.tile})", us, 4 * touched * d * ff + T * k * 2 * (d + ff), 4.0 * T * k * d * ff, "fb_linear_indexed")
    us = timed(20, copies, lambda i: ops.grouped(act, down[i], r, y))
    row("fb_dense_grouped down", us, 2 * touched * d * ff + T * k * 2 * (d + ff), 2.0 * T * k * d * ff, "fb_linear_indexed")
    res, out, one = f32(T, d), f32(T, d), f32_ones(dev, d)
    us = timed(40, 1, lambda i: ops.add_norm(res, out, h, one, h, one, y, r, one, 1.0, 1e-5, x[:T]))
    row("fb_add_norm", us, T * d * (8 + 6 + 2 * k), like="fb_rmsnorm")
    table, ids = bf(s["vocab"], d), torch.arange(T, device=dev, dtype=torch.int32)
    us = timed(40, 1, lambda i: ops.embed(table, ids, table, ids, out))
    row("fb_embed", us, T * d * 8, like="fb_gather_rows")
    return rows


def vunadra_kernels(rt, s, T, ctx, peaks):
    """Each kernel of the Vunadra layers, as design_kernels does it."""
    import torch
    from ferrite_b200 import _lib, ops
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    f32 = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen)
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.bfloat16).normal_(0, 1, generator=gen)
    ones = lambda n: f32_ones(dev, n)
    rows, prompt = [], ctx == 0
    d, H, G, dim, vd, E, k, ff, dff, rank, rd, window, taps = (s[n] for n in ("width", "heads", "kv", "dim", "vdim", "experts", "top", "ff", "dense", "kv_rank", "rot_dim", "window", "conv"))

    def row(name, us, nbytes, flops=0.0, like=None):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)} | ({"like": like} if like else {}))

    def dense(name, K, N, batch=1, kind=_lib.DENSE_NONE, out_dtype=torch.bfloat16, like="fb_linear"):
        copies = max(1, min(16, int(3e8 // (2 * batch * K * N))))
        ws, x, cols = [bf(batch, N, K) for _ in range(copies)], bf(T, batch, K).permute(1, 0, 2), N // 2 if kind == _lib.DENSE_GEGLU else N
        out, b = torch.empty(T, batch, cols, device=dev, dtype=out_dtype).permute(1, 0, 2), ones(N)
        extra = dict(gate_bias=b.data_ptr(), up_bias=b.data_ptr()) if kind == _lib.DENSE_GEGLU else {}
        us = timed(40, copies, lambda i: ops.dense(x, ws[i].transpose(1, 2), out, True, kind, **extra))
        row(f"fb_dense {name} {batch}x[{K}, {N}]" if batch > 1 else f"fb_dense {name} [{K}, {N}]", us, 2 * batch * K * N + 2 * T * batch * K + out.element_size() * T * batch * cols,
            2.0 * T * batch * K * N, like)

    qkv, qk, W = (H + G) * dim + G * vd, (H + G) * dim, rank + rd
    dense("pass start", 2 * d, d, out_dtype=torch.float32)
    dense("q, k, v", d, qkv, out_dtype=torch.float32)
    dense("q, k", d, qk, out_dtype=torch.float32)
    dense("q, dkv", d, H * (dim + rd) + W, out_dtype=torch.float32)
    dense("uk by head", dim, rank, H)
    dense("uv by head", rank, vd, H)
    dense("o", H * vd, d)
    dense("gate_up, gelu", d, 2 * dff, 1, _lib.DENSE_GEGLU)
    dense("down", dff, d)
    dense("router", d, E + s["identity"], out_dtype=torch.float32, like="router")
    dense("head", d, s["vocab"], out_dtype=torch.float32)

    keys = T if prompt else ctx
    part, seqs = keys + -keys % 64, 1 if prompt else T
    caches = [bf(G, seqs * part, dim + vd) for _ in range(4)]
    last = torch.arange(T, device=dev, dtype=torch.int32) if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    base = torch.arange(T, device=dev, dtype=torch.int32) * part
    at, q, o, first = (last if prompt else base + last), bf(T, H * dim), bf(T, H * vd), None if prompt else base
    joint, state, turn = f32(T, qkv), f32(seqs, taps - 1, qkv), (torch.ones(dim // 2, device=dev, dtype=torch.float64), dim, 1.0)
    conv = f32(taps, qkv)
    us = timed(40, 1, lambda i: ops.heads_put(joint, H, G, dim, vd, at, caches[0], q, rotation=turn, places=last, conv=conv, state=state, dead=-1))
    row("fb_heads_put, convolution, turn", us, T * 6 * qkv + (seqs * 2 * (taps - 1) + taps) * qkv * 4, like="fb_rope_kv_write")
    us = timed(40, 1, lambda i: ops.heads_put(joint, H, G, dim, dim, at, caches[0], q, ones(qk), ones(H * dim), ones(G * dim), 1e-5, norm_all=True, keys_are_values=True, rotation=turn, places=last))
    row("fb_heads_put, joint norms, turn, keys as values", us, T * (4 * qk + 2 * (qk + G * dim)), like="fb_rope_kv_write")
    within = min(window, keys)
    seen = within * (within + 1) / 2 + max(0, T - within) * within if prompt else T * within
    pairs = T * (T + 1) / 2 if prompt else T * ctx
    us = timed(20, 4, lambda i: ops.heads_attention(q, caches[i], first, last, H, vd, 0.1, keys, prompt, out=o))
    row("fb_heads_attention", us, 2 * (seqs * keys * G * (dim + vd) + T * H * (dim + vd)), 2.0 * pairs * H * (dim + vd), "attention")
    us = timed(20, 4, lambda i: ops.heads_attention(q, caches[i], first, last, H, vd, 0.1, keys, prompt, out=o, window=window, softcap=30.0))
    row(f"fb_heads_attention, window of {window}, capped", us, 2 * (seqs * (keys if prompt else within) * G * (dim + vd) + T * H * (dim + vd)), 2.0 * seen * H * (dim + vd), "attention")
    us = timed(20, 4, lambda i: ops.heads_attention(q, caches[i], first, last, H, vd, 0.1, keys, prompt, out=o, softcap=30.0))
    row("fb_heads_attention, no window, capped", us, 2 * (seqs * keys * G * (dim + vd) + T * H * (dim + vd)), 2.0 * pairs * H * (dim + vd), "attention")
    lcaches, lq, lo = [bf(seqs * part, W) for _ in range(4)], bf(T, H * W), bf(T, H * rank)
    down, plain, freq = f32(T, H * (dim + rd) + W), bf(T, H * dim), torch.ones(rd // 2, device=dev, dtype=torch.float64)
    turned = lq.view(T, H, W).permute(1, 0, 2)[:, :, rank:]
    us = timed(40, 1, lambda i: ops.latent_put(down, 0, rank, rd, rd, None, ones(rank), 1e-5, freq, 1.0, last, at, lcaches[0], plain, H, dim, turned))
    row("fb_latent_put, queries", us, T * (H * (dim + rd) + W) * 6, like="fb_rope_kv_write")
    us = timed(20, 4, lambda i: ops.latent_attention(lq, lcaches[i], first, last, H, rank, 0.1, None, keys, prompt, out=lo, window=window))
    row(f"fb_latent_attention, window of {window}", us, 2 * (seqs * (keys if prompt else within) * W + T * H * (W + rank)), 2.0 * seen * H * (W + rank), "attention")
    if prompt:  # (the same attention with keys and values made first)
        row("fb_latent_attention, counted as keys and values of a head", us, 0, 2.0 * seen * H * (dim + rd + vd), "attention")

    n = E + s["identity"]
    logits = f32(T, n)
    us = timed(40, 1, lambda i: ops.route(logits, n, k, ones(n), True, s["identity"], 1.0))
    row("fb_route", us, T * (4 * n + 12 * k), like="fb_topk and fb_touched (fb_group)")
    r = ops.route(logits, n, k, None, True, s["identity"], 1.0)
    ids = [e for e in r.ids.cpu().reshape(-1).tolist() if e < E]
    touched, live, choices = len(set(ids)), int(r.live), len(ids)
    copies = max(1, min(4, int(3e8 // (6 * touched * d * ff)) + 1))
    gate_up, down, h = [bf(E, 2 * ff, d).transpose(1, 2) for _ in range(copies)], [bf(E, d, ff).transpose(1, 2) for _ in range(copies)], bf(T, d)
    x, act, y = bf(r.tiles * r.tile, d), bf(r.tiles * r.tile, ff), bf(r.tiles * r.tile, d)
    if not r.shared:
        us = timed(20, 1, lambda i: ops.spread_rows(h, r, x))
        row("fb_spread_rows", us, 2 * (T + choices) * d, like="fb_gather_rows")
    us = timed(20, copies, lambda i: ops.grouped(h if r.shared else x, gate_up[i], r, act, _lib.DENSE_GLU, r.shared, limit=7.0, slope=1.702))
    row(f"fb_dense_grouped gate_up, clamped unit ({touched} experts, {live} tiles of {r.tile})", us, 4 * touched * d * ff + choices * 2 * (d + ff), 4.0 * choices * d * ff, "fb_linear_indexed")
    us = timed(20, copies, lambda i: ops.grouped(act, down[i], r, y))
    row("fb_dense_grouped down", us, 2 * touched * d * ff + choices * 2 * (d + ff), 2.0 * choices * d * ff, "fb_linear_indexed")
    res, out, one = f32(T, d), f32(T, d), ones(d)
    us = timed(40, 1, lambda i: ops.add_norm(res, out, chosen=y, routes=r, w=one, eps=1e-5, h=h, own=h))
    row("fb_add_norm, chosen rows", us, T * d * (8 + 2 + 2 * k), like="fb_rmsnorm")
    us = timed(40, 1, lambda i: ops.add_norm(res, out, o[:, :d] if H * vd >= d else h, w=one, eps=1e-5, h=h, mixer_bias=one))
    row("fb_add_norm, bias", us, T * d * (8 + 2 + 2), like="fb_rmsnorm")
    return rows


def ronavik_kernels(rt, s, T, ctx, peaks):
    """Each kernel of the Ronavik layers, as design_kernels does it; beside the state space's scan the fixed decay's over as many heads of that size."""
    import torch
    from ferrite_b200 import _lib, ops
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    f32 = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.float32).normal_(0, 1, generator=gen)
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.bfloat16).normal_(0, 1, generator=gen)
    rows, prompt = [], ctx == 0
    d, H, G, dim, vd, W, blocks, taps = (s[n] for n in ("width", "heads", "kv", "dim", "vdim", "lru", "blocks", "conv"))
    SH, P, N, SG, E, k, ff = (s[n] for n in ("ssm_heads", "ssm_vdim", "state", "groups", "experts", "top", "ff"))
    inner, n = SH * P, (H + G) * dim + G * vd
    wide = inner + 2 * SG * N

    def row(name, us, nbytes, flops=0.0, like=None):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)} | ({"like": like} if like else {}))

    def dense(name, K, N, out_dtype=torch.bfloat16, batch=1):
        copies = max(1, min(16, int(3e8 // (2 * batch * K * N))))
        ws, x = [bf(batch, N, K) for _ in range(copies)], bf(T, batch, K).permute(1, 0, 2)
        out = torch.empty(T, batch, N + -N % 8, device=dev, dtype=out_dtype).permute(1, 0, 2)[:, :, :N]
        us = timed(40, copies, lambda i: ops.dense(x, ws[i].transpose(1, 2), out, True))
        row(f"fb_dense {name} " + (f"{batch}x" if batch > 1 else "") + f"[{K}, {N}]", us, batch * (2 * K * N + 2 * T * K + out.element_size() * T * N), 2.0 * T * batch * K * N, "fb_linear")

    dense("parallel: gate, q, k, v, y, x", d, d + n + 2 * W, torch.float32)
    dense("mamba2: gate, z, x, B, C, dt", d, d + inner + wide + SH, torch.float32)
    dense("gates by block", W // blocks, 2 * W // blocks, torch.float32, blocks)
    dense("parallel o", H * vd + W, d)
    dense("mamba2 o", inner, d)
    dense("gate, router", d, d + E, torch.float32)
    dense("head", d, s["vocab"], torch.float32)

    places = torch.arange(T, device=dev, dtype=torch.int32) if prompt else torch.full((T,), ctx - 1, device=dev, dtype=torch.int32)
    slots, keys, dead = 1 if prompt else T, T if prompt else ctx, -1
    part = keys + -keys % 64
    base = torch.arange(T, device=dev, dtype=torch.int32) * part
    pairs = T * (T + 1) / 2 if prompt else T * ctx
    for v in (vd, 2 * vd):
        caches, m = [bf(G, slots * part, dim + v) for _ in range(4)], (H + G) * dim + G * v
        joint, q, both = f32(T, d + m + 2 * W), bf(T, H * dim), bf(T, H * v + W)
        us = timed(40, 1, lambda i: ops.heads_put(joint[:, d:d + m], H, G, dim, v, places if prompt else base + places, caches[0], q, q_norm=f32_ones(dev, dim), k_norm=f32_ones(dev, dim), eps=1e-5, places=places,
                                                  temperature=(0.1, 8192.0)))
        if v == vd:
            row("fb_heads_put, temperature", us, T * 6 * m, like="fb_rope_kv_write")
        us = timed(20, 4, lambda i: ops.heads_attention(q, caches[i], None if prompt else base, places, H, v, 0.1, keys, prompt, key_bias=f32_ones(dev, H), out=both[:, :H * v]))
        row("fb_heads_attention by sigmoids" + ("" if v == vd else f", values of {v} columns"), us, 2 * (slots * keys * G * (dim + v) + T * H * (dim + v)), 2.0 * pairs * H * (dim + v), "attention")

    joint, u, gates = f32(T, d + n + 2 * W), bf(T, W), f32(T, 2 * W)
    x, y = joint[:, d + n + W:d + n + 2 * W], joint[:, d + n:d + n + W]
    conv, w = f32(slots, taps - 1, max(W, wide)), f32(taps, max(W, wide))
    us = timed(40, 1, lambda i: ops.short_conv(x, w.view(-1)[:taps * W].view(taps, W), u, places, dead, conv.view(-1)[:slots * (taps - 1) * W].view(slots, taps - 1, W), f32_ones(dev, W), f32_ones(dev, W)))
    row("fb_short_conv, recurrence", us, T * W * 6 + slots * (taps - 1) * W * 8, like="fb_rope_kv_write")
    state = f32(slots, 1, W)
    us = timed(40, 1, lambda i: ops.lru_scan(u, gates, y, both[:, -W:], f32_ones(dev, W), -8.0, blocks, places, dead, state, f32_ones(dev, 2 * W), f32_ones(dev, W)))
    row("fb_lru_scan", us, T * W * 16 + slots * W * 8, like="fb_decay_scan")

    joint, xbc, out = f32(T, d + inner + wide + SH + -SH % 8), bf(T, wide), f32(T, inner)
    us = timed(40, 1, lambda i: ops.short_conv(joint[:, d + inner:d + inner + wide], w.view(-1)[:taps * wide].view(taps, wide), xbc, places, dead, conv.view(-1)[:slots * (taps - 1) * wide].view(slots, taps - 1, wide),
                                               f32_ones(dev, wide), None, True))
    row("fb_short_conv, state space", us, T * wide * 6 + slots * (taps - 1) * wide * 8, like="fb_rope_kv_write")
    step, states, low = joint[:, d + inner + wide:d + inner + wide + SH], [f32(slots, SH * N, P) for _ in range(1 if prompt else 4)], f32_ones(dev, SH) * -2
    us = timed(20, len(states), lambda i: ops.selective_scan(xbc, SH, SG, N, P, step, low, low, low, places, dead, states[i], out))
    row("fb_selective_scan", us, T * (2 * wide + 4 * SH + 4 * inner) + slots * SH * N * P * 8, 2.0 * T * SH * 2 * N * P, "fb_decay_scan")
    qkv, decay = bf(T, SH * (2 * N + P)), torch.full((SH,), 0.95, device=dev)
    us = timed(20, len(states), lambda i: ops.decay_scan(qkv, SH, N, P, decay, places, dead, states[i], out))
    row("fb_decay_scan, the fixed decay's", us, T * (2 * SH * (2 * N + P) + 4 * inner) + slots * SH * N * P * 8, 2.0 * T * SH * 2 * N * P)
    h = bf(T, inner)
    us = timed(40, 1, lambda i: ops.gated_rmsnorm(out, joint[:, d:d + inner], f32_ones(dev, inner), 1e-5, h, True, SG))
    row("fb_gated_rmsnorm, gate before, in parts", us, T * inner * 10, like="fb_rmsnorm")

    logits = f32(T, E)
    us = timed(40, 1, lambda i: ops.route(logits, E, k, None, "sigmoid", as_scored=True, on_input=True))
    row("fb_route, sigmoids", us, T * (4 * E + 12 * k), like="fb_topk and fb_touched (fb_group)")
    r = ops.route(logits, E, k, None, "sigmoid", as_scored=True, on_input=True)
    touched, live = len(set(r.ids.cpu().reshape(-1).tolist())), int(r.live)
    copies = max(1, min(4, int(3e8 // (4 * touched * d * ff)) + 1))
    up, down, h = [bf(E, ff, d).transpose(1, 2) for _ in range(copies)], [bf(E, d, ff).transpose(1, 2) for _ in range(copies)], bf(T, d)
    x, act, y = bf(r.tiles * r.tile, d), bf(r.tiles * r.tile, ff), bf(r.tiles * r.tile, d)
    if not r.shared:
        us = timed(20, 1, lambda i: ops.spread_rows(h, r, x))
        row("fb_spread_rows", us, 2 * T * (k + 1) * d, like="fb_gather_rows")
    us = timed(20, copies, lambda i: ops.grouped(h if r.shared else x, up[i], r, act, _lib.DENSE_RELU2, r.shared, row_scale=r.row_weights.data_ptr()))
    row(f"fb_dense_grouped up, squared ReLU ({touched} experts, {live} tiles of {r.tile})", us, 2 * touched * d * ff + T * k * 2 * (d + ff), 2.0 * T * k * d * ff, "fb_linear_indexed")
    us = timed(20, copies, lambda i: ops.grouped(act, down[i], r, y))
    row("fb_dense_grouped down", us, 2 * touched * d * ff + T * k * 2 * (d + ff), 2.0 * T * k * d * ff, "fb_linear_indexed")
    res, sums, one, gate = f32(T, d), f32(T, d), f32_ones(dev, d), f32(T, d + E + -E % 8)
    for what, more in (("mixer", dict(mixer=h)), ("chosen rows", dict(chosen=y, routes=r))):
        us = timed(40, 1, lambda i: ops.add_norm(res, sums, w=one, eps=1e-5, h=x[:T], gate=gate[:, :d], gate_bias=one, post=one, **more))
        row(f"fb_add_norm, {what}, gated and normed", us, T * d * (8 + 4 + 2 + 2 * (1 if what == "mixer" else k)), like="fb_rmsnorm")
    return rows


def llama_expert_kernels(rt, s, T, peaks):
    """The Llama mixture's own kernels at the same size (bfp8 experts): its router's and its experts', decode or prompt."""
    import torch
    from ferrite_b200 import ops
    from ferrite_b200.llama import glu
    from ferrite_b200.tensor import Tensor
    dev, gen = rt.device, torch.Generator(device=rt.device).manual_seed(0)
    d, E, k, ff, rows = s["width"], s["experts"], s["top"], s["ff"], []
    bf = lambda *shape: torch.empty(*shape, device=dev, dtype=torch.bfloat16).normal_(0, 1, generator=gen)

    def row(name, us, nbytes, flops=0.0):
        floor = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3)})

    logits = Tensor(rt, T, E, dtype="fp32", buf=torch.empty(1, T, E, device=dev).normal_(0, 1, generator=gen))
    values, ids = logits.topk(k)
    w = values.softmax().bfloat16().realize()
    touched = len(set(ids.numpy().reshape(-1).tolist()))

    def picks():
        v, i = logits.topk(k)
        u = v.softmax().bfloat16().realize()
        return i.touched(E, u) if T <= 128 else i.group(E)
    row("fb_topk, softmax and " + ("fb_touched" if T <= 128 else "fb_group"), timed(20, 1, lambda i: picks()), T * (4 * E + 12 * k))
    pack = lambda K, N: Tensor(rt, K, N, batch=E, dtype="bfp8", packed=ops.quantize(bf(E, K, N), "bfp8"))
    gate_up, down, h = pack(d, 2 * ff), pack(ff, d), Tensor(rt, T, d, buf=bf(1, T, d))
    up_bytes, down_bytes = 1.0625 * touched * 2 * d * ff, 1.0625 * touched * d * ff
    if T <= 128:
        index, weights = ids.touched(E, w)
        act, n = bf(T, index.rows * ff), index.rows
        idx, out = index.buf.reshape(-1), bf(T, d)
        us = timed(20, 1, lambda i: ops.linear_indexed(h.buf[0], gate_up.packed, idx, act, out_slot_stride=ff, epilogue="swiglu", row_scale=weights.buf))
        row(f"fb_linear_indexed gate_up, swiglu ({touched} experts)", us, up_bytes + T * k * 2 * (d + ff), 4.0 * T * k * d * ff)
        us = timed(20, 1, lambda i: ops.linear_indexed(act, down.packed, idx, out, sum_slots=True))
        row("fb_linear_indexed down, summed", us, down_bytes + T * k * 2 * (d + ff), 2.0 * T * k * d * ff)
    else:
        order, tiles, _ = ids.group(E)
        x = Tensor(rt, 32, d, batch=tiles.rows, buf=bf(tiles.rows, 32, d))
        us = timed(4, 1, lambda i: x.matmul(gate_up, index=tiles).realize())
        row(f"fb_linear_indexed gate_up ({touched} experts, tiles of 32)", us, up_bytes + T * k * 2 * (d + 2 * ff), 4.0 * T * k * d * ff)
        y = x.matmul(gate_up, index=tiles).realize()
        us = timed(4, 1, lambda i: glu(y[:, :, :ff], y[:, :, ff:]).realize())
        row("fb_elementwise silu, times", us, T * k * 6 * ff)
        z = glu(y[:, :, :ff], y[:, :, ff:]).realize()
        us = timed(4, 1, lambda i: z.matmul(down, index=tiles).realize())
        row("fb_linear_indexed down", us, down_bytes + T * k * 2 * (d + ff), 2.0 * T * k * d * ff)
    return rows


def run_design(args):
    """--design: one JSON line a size."""
    import torch
    from ferrite_b200 import llama, models
    from ferrite_b200.tensor import Runtime
    name, _, size = args.design.partition(":")
    designs = {"binutar": (DESIGN_SIZES, design_models, design_kernels), "labepel": (LABEPEL_SIZES, labepel_models, labepel_kernels), "vunadra": (VUNADRA_SIZES, vunadra_models, vunadra_kernels),
               "ronavik": (RONAVIK_SIZES, ronavik_models, ronavik_kernels)}
    assert name in designs and args.gpus == 1, "--design " + " or ".join(f"{n}[:SIZE]" for n in designs) + ", one GPU"
    sizes, make, kernels = designs[name]
    rt, (peaks, kind), family = Runtime(0), measured_peaks(), models.module(name)
    S, ctx, prompt = 32, 2048, 2048
    for key in [size] if size else sizes:
        s = sizes[key]
        clocks = Clocks(0)
        clocks.start()
        line = {"design": name, "size": key, "shape": s, "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": kind}, "weights": "random"}
        b, l = make(s, ctx + 256)
        for c, module, mode in ((b, family, "bf16"), (b, family, "bfp8"), (l, llama, "bfp8")):
            line[f"{c.family} {mode}"] = design_steps(rt, c, module.precision(c, mode), S, ctx, prompt, args.steps)
            torch.cuda.empty_cache()
        for what, T, at in (("decode", S, ctx), ("prefill", prompt, 0)):
            own = kernels(rt, s, T, at, peaks)
            torch.cuda.empty_cache()
            like = llama_kernels(rt, s, T, at, peaks) + (llama_expert_kernels(rt, s, T, peaks) if "experts" in s else [])
            line["kernels " + what] = {name: own, "llama": like}
            torch.cuda.empty_cache()
        line["clocks"] = clocks.summary()
        print(json.dumps(line), flush=True)


def matmul_sweep(device, peak_gbs, calls=200):
    """the isolated block-float matmul, RMSNorm prologue and SwiGLU epilogue fused, K = 4096,
    M in {1, 8, 32, 128}, N in {4096, 14336}, bfp8 and bfp4.  `calls` back-to-back calls (one recorded graph) rotate
    through distinct weight buffers that together exceed L2 several times, so every call streams its matrix from HBM.
    Algorithmic bytes per call: the packed matrix, the activations in, the result out, the norm's weight."""
    import torch
    from ferrite_b200 import ops
    K, rows, gen = 4096, [], torch.Generator(device=device).manual_seed(0)
    g = (1 + 0.1 * torch.randn(K, device=device, generator=gen)).bfloat16()
    for fmt, per_value in (("bfp8", 1.0625), ("bfp4", 0.5625)):
        for N in (4096, 14336):
            copies = min(48, -(-(512 << 20) // int(K * N * per_value)))
            ws = [ops.quantize((torch.randn(K, N, device=device, generator=gen) * 0.02).bfloat16(), fmt) for _ in range(copies)]
            for M in (1, 8, 32, 128):
                x = torch.randn(M, K, device=device, generator=gen).bfloat16()
                out = torch.empty(M, N // 2, device=device, dtype=torch.bfloat16)
                for i in range(3):
                    ops.linear(x, ws[i % copies], out=out, norm_w=g, eps=1e-5, epilogue="swiglu")
                torch.cuda.synchronize()
                graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(graph):
                    for i in range(calls):
                        ops.linear(x, ws[i % copies], out=out, norm_w=g, eps=1e-5, epilogue="swiglu")
                graph.replay()
                torch.cuda.synchronize()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                graph.replay()
                e1.record()
                torch.cuda.synchronize()
                us = e0.elapsed_time(e1) * 1e3 / calls
                nbytes = K * N * per_value + 2 * M * K + 2 * M * (N // 2) + 2 * K
                rows.append({"fmt": fmt, "M": M, "N": N, "us": round(us, 2), "GB/s": round(nbytes / us / 1e3, 1),
                             "frac": round(nbytes / us / 1e3 / peak_gbs, 3)})
            del ws
            torch.cuda.empty_cache()
    return {"what": "RMSNorm + [M,4096]x[4096,N] + SwiGLU, %d calls rotating weight copies > L2" % calls, "peak_GB/s": peak_gbs, "rows": rows}


def cpu_sample(args, seconds):
    """One decode step of ONE block plus the output layer of the workload on this box's host cores, timed, and scaled to
    the model's block count.  It runs the reference's OWN numpy code (models/llama.py: around, layer, rms - the numpy
    branch its `fns` picks) when oracle/_ref holds it (oracle/make_ref.py put it there from a checkout; kind
    "reference"), else the restatement under oracle/ (kind "port").  Weights are quantised by the C restatement."""
    from oracle import build as obuild
    from oracle import llama as ollama
    from oracle import make_ref
    ref = make_ref.modules()
    wl = WORKLOADS[args.workload]
    fields = {k: v for k, v in wl["model"].items() if k != "tied"} | dict(places=wl["context"] + 64)
    layers = args.layers or fields["layers"]
    oc = ollama.model(**fields | dict(layers=1))
    c = ref[0].model(**{k: v for k, v in fields.items() if k != "qk_norm"} | dict(layers=1)) if ref else oc
    S, ctx = wl["sequences"], wl["context"]
    rng = np.random.default_rng(0)
    ctxs = [int(v) for v in rng.integers(wl["ragged"][0], wl["ragged"][1] + 1, S)] if wl.get("ragged") else [ctx] * S
    hd, nh = ollama.head(oc), oc.heads + 2 * oc.kv
    fmt = "bfp8" if wl["mode"] == "experts" else wl["mode"]
    q = lambda *shape, f=fmt: obuild.bfp_values(rng.standard_normal(shape, dtype=np.float32) * np.float32(0.02), f)
    w = {"layers.0.input_layernorm": np.ones((1, oc.dim), np.float32), "layers.0.post_attention_layernorm": np.ones((1, oc.dim), np.float32),
         "layers.0.qkv_proj": q(oc.dim, nh * hd), "layers.0.o_proj": q(oc.heads * hd, oc.dim), "norm": np.ones((1, oc.dim), np.float32)}
    if getattr(oc, "experts", 0):
        ef = "bfp4" if wl["mode"] == "experts" else fmt
        w["layers.0.router"] = (rng.standard_normal((oc.dim, oc.experts), dtype=np.float32) * np.float32(0.02))
        w["layers.0.experts.gate_up"] = np.stack([q(oc.dim, 2 * oc.moe, f=ef) for _ in range(oc.experts)])
        w["layers.0.experts.down"] = np.stack([q(oc.moe, oc.dim, f=ef) for _ in range(oc.experts)])
        if wl["model"].get("qk_norm"):
            w["layers.0.qk_norm"] = np.ones((nh, 1, hd), np.float32)
            w["layers.0.qk_on"] = np.array([1.0] * (oc.heads + oc.kv) + [0.0] * oc.kv, np.float32).reshape(nh, 1, 1)
    else:
        w["layers.0.gate_up_proj"], w["layers.0.down_proj"] = q(oc.dim, 2 * oc.ffn), q(oc.ffn, oc.dim)
    w["embed"] = (rng.standard_normal((oc.vocab, oc.dim), dtype=np.float32) * np.float32(0.02))
    w["embed.T"] = obuild.bfp_values(np.ascontiguousarray(w["embed"].T), fmt)
    if ref:
        w["cos"], w["sin"], w["turn"] = ref[0].rotary(c, c.places)
    else:
        w["cos"], w["sin"] = ollama.rotary(oc, oc.places)
    part = ctx + 64
    caches = [np.zeros((2 * oc.kv, S * part, hd))]  # np.zeros: float64, as the reference's kv_cache(c, size, np.zeros)
    caches[0][:, :, :] = rng.standard_normal(caches[0].shape)
    ids = [int(v) for v in rng.integers(0, oc.vocab, S)]
    slots = S if S > 1 else None
    threads = blas_threads()
    times, place = [], 0
    start = time.perf_counter()
    while not times or (time.perf_counter() - start < seconds and len(times) < 16):
        t0 = time.perf_counter()
        x = w["embed"][ids]
        places, size = ([v + place for v in ctxs] if slots else [ctx + place]), (S * part if slots else part)
        if ref:
            rows, rotary, mask, _, live = ref[0].around(w, c, places, size, slots)
        else:
            rows, cos, sin, mask, live = ollama.around(w, oc, places, size, slots)
        t_in = time.perf_counter()
        if ref:
            x = ref[0].layer(x, ref[1].block(w, "layers.0."), c, rotary, mask, caches[0], rows, 0, False, live, None, slots)
        else:
            x = ollama.layer(x, ollama.block(w, "layers.0."), oc, cos, sin, mask, caches[0], rows, live, slots)
        t_layer = time.perf_counter()
        logits = (ref[0].rms(x, w["norm"], c) if ref else ollama.rms(x, w["norm"], oc.eps)) @ w["embed.T"]
        picks = logits.argmax(-1)
        t_head = time.perf_counter()
        times.append(((t_in - t0) + (t_head - t_layer), t_layer - t_in))
        place += 1
    rest, layer = np.median([t[0] for t in times]), np.median([t[1] for t in times])
    step_seconds = rest + layers * layer
    return {"value": S / step_seconds, "unit": "tokens/s", "cores": os.cpu_count(), "blas_threads": threads, "kind": "reference" if ref else "port",
            "sample": f"{len(times)} decode steps of 1 of {layers} blocks plus embedding and output layer, "
                      + ("the reference's own models/llama.py numpy branch" if ref else "the numpy restatement of the reference's CPU path")
                      + " (float32 weights, float64 KV cache as the reference keeps it); block time x " + f"{layers} + the rest",
            "seconds_per_step_scaled": step_seconds}


def blas_threads():
    """The threads numpy's BLAS uses (what the CPU legs' matmuls run on), pinned to the host's cores where a launcher
    set it to one (torch.distributed.run exports OMP_NUM_THREADS=1 to its workers)."""
    try:
        from threadpoolctl import threadpool_info, threadpool_limits
        want = os.cpu_count() or 1
        threadpool_limits(want)
        return max([p.get("num_threads", 1) for p in threadpool_info()] or [1])
    except Exception:  # noqa: BLE001  (threadpoolctl missing: numpy's default)
        return None


def cpu_baseline(args, sample_seconds):
    return cpu_sample(args, sample_seconds)


def run_reference(args):
    """The reference arm: the reference's CPU path (its numpy branch, restated under oracle/) on this box's host cores."""
    if int(os.environ.get("RANK", 0)) != 0:
        return
    wl = WORKLOADS[args.workload]
    base = cpu_sample(args, seconds=min(120, 4 * max(args.steps, 1)))
    S = wl["sequences"]
    line = {"impl": "reference", "metric": "decode tokens/s", "value": base["value"], "unit": "tokens/s", "n_gpus": args.gpus, "steps": args.steps,
            "warmup": args.warmup, "ms_per_step": 1e3 * S / base["value"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
            "dtype": "f32", "data": "synthetic",
            "config": {"workload": wl["name"], "layers": args.layers or wl["model"]["layers"], "parallelism": "host cores"},
            "cpu_baseline": base, "e2e": {"value": base["value"], "unit": "tokens/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0}}
    print(json.dumps(line), flush=True)


if __name__ == "__main__":
    a = parse()
    if a.matmul:
        one_matmul(a.matmul)
    elif a.attend:
        one_attention(a.attend)
    elif a.design:
        run_design(a)
    else:
        run_reference(a) if a.impl == "reference" else run_ferrite(a)
