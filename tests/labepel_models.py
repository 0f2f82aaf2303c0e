"""Small Labepel configurations and checkpoints for the tests: random weights, made so that the parts that random weights
would hide are seen in the logits - attention that is peaked, values that are mixed by much, biases that matter - and so that
no choice of experts is a close call: each token's embedding says in columns of its own, which nothing adds to, how much it
likes each expert."""
import numpy as np

from binutar_models import error, save  # noqa: F401  (a checkpoint is written, and logits are compared, as for the other design)
from oracle import labepel as oracle


def attention(heads=4, kv_heads=2, dim=24, vdim=40, size=20, scale=0.22, v_mix=True, ff=48, experts=6, top=2, shared=40):
    mlp = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff)) | (dict(shared=dict(ff=shared)) if shared else {}) if ff else None
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=size), scale=scale, v_mix=v_mix), mlp=mlp)


def config(width, vocab, layers, eps=1e-5, positions=700):
    return dict(architecture="Labepel", vocab=vocab, width=width, norm=dict(eps=eps), max_positions=positions, layers=layers)


# name -> config.json: spans of several sizes, layers without a feed-forward, without mixed values and (the first that mixes is
# then a later one) without a shared expert; sizes that only the general kernels take (odd); values that are often equal or 1;
# more query heads a key head than a tile has rows, wide heads, many experts
CONFIGS = {
    "mixed": config(96, 200, [attention(v_mix=False), attention(heads=8, dim=16, size=33), attention(kv_heads=4, vdim=20, size=64, ff=None), attention(size=7, shared=None, top=3)]),
    "odd": config(60, 131, [attention(heads=3, kv_heads=1, dim=9, vdim=7, size=5, ff=13, experts=5, top=3, shared=11), attention(heads=6, kv_heads=1, dim=11, vdim=7, size=17, ff=21, experts=7, top=1, shared=None)], 1e-3),
    "ones": config(64, 96, [attention(heads=1, kv_heads=1, dim=64, vdim=64, size=1, ff=64, experts=1, top=1, shared=64), attention(heads=1, kv_heads=1, dim=64, vdim=64, size=600, ff=64, experts=1, top=1, shared=64)], 1e-6),
    "wide": config(128, 320, [attention(heads=20, kv_heads=1, dim=136, vdim=16, size=100, scale=0.1, experts=40, top=8, ff=32), attention(heads=2, kv_heads=1, dim=32, vdim=16, size=48, experts=40, top=40, ff=16)]),
    "spans": config(64, 128, [attention(heads=4, kv_heads=4, dim=32, vdim=32, size=n, ff=32, experts=4, top=1, shared=32) for n in (64, 65, 16)]),
}


def weights(cfg, seed=0):
    """{tensor name: float32 array of bf16 values} of a configuration."""
    rng, out, d = np.random.default_rng(seed), {}, cfg["width"]
    n = max([e["mlp"]["router"]["experts"] for e in cfg["layers"] if e["mlp"]], default=0)  # the columns that choose experts: 0 .. n - 1
    for name, shape in oracle.tensors(cfg).items():
        if name.endswith("vmix"):
            x = rng.uniform(0.25, 0.6, shape)
        elif name.endswith((".q.norm", ".k.norm")):
            x = rng.normal(1.6, 0.3, shape)
        elif name.endswith("norm1") or name == "final.norm":
            x = rng.normal(0, 0.2, shape)
            x[:n] = 0
        elif name.endswith((".ls1", ".ls2")):
            x = rng.normal(0.7, 0.2, shape)
            x[:n] = 0
        elif name.endswith("router.b"):
            x = rng.uniform(-0.15, 0.15, shape)
        elif name.endswith(".b"):
            x = rng.normal(0, 0.4, shape)
        elif name == "embed":
            x = rng.normal(0, 1.0, shape)
            x[:, :n] = np.argsort(rng.random((shape[0], n)), axis=1) * (2.0 / n) if n else x[:, :n]
        elif name == "pos":
            x = rng.normal(0, 0.7, shape)
            x[:, :n] = 0
        elif name.endswith("router"):
            x = np.zeros(shape)
            x[:, n:] = rng.normal(0, 0.05 * d ** -0.5, (shape[0], d - n))
            x[np.arange(shape[0]), np.arange(shape[0])] = n
        else:
            x = rng.normal(0, 1.2 * shape[1] ** -0.5, shape)
        bits = np.asarray(x, np.float32).reshape(-1).view(np.uint32)
        bits = ((bits + (0x7FFF + (bits >> 16 & 1))) >> 16 << 16).astype(np.uint32)
        out[name] = bits.view(np.float32).reshape(shape)
    return out


class Alone:
    """The oracle's logits of one token sequence, with what it needs kept between calls."""

    def __init__(self, cfg, w):
        self.cfg, self.w, self.caches, self.at = cfg, w, oracle.caches(cfg), 0

    def __call__(self, ids):
        out = oracle.forward(ids, self.at, self.w, self.cfg, self.caches)
        self.at += len(ids)
        return out


def greedy(cfg, w, prompt, n):
    """A greedy continuation."""
    run, made = Alone(cfg, w), []
    out = run(prompt)
    for _ in range(n):
        made.append(int(out[-1].argmax()))
        out = run(made[-1:])
    return made
