"""Small Ronavik configurations and checkpoints for the tests: random weights, made so that the parts that random weights would
hide are seen in the logits - keys that stand out, convolutions that matter, states that remember some tens of tokens - and so that no
choice of experts is a close call: each token's embedding says in columns of its own, which places and layers leave as they are, how
much it likes each expert."""
import numpy as np

from binutar_models import error, save  # noqa: F401  (a checkpoint is written, and logits are compared, as for the other design)
from oracle import ronavik as oracle


def moe(experts=6, top=2, ff=48):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def mamba2(heads=6, vdim=24, state=32, groups=2, conv=4, norm_groups=3, mlp=None):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups), mlp=mlp)


def parallel(heads=6, kv_heads=2, dim=32, vdim=40, scale=0.2, coef=0.4, every=10, width=64, blocks=4, conv=3, left=0.7, right=1.2, mlp=None):
    return dict(type="parallel", mixer=dict(left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, q_temp=dict(coef=coef, every=every)),
                                            right=dict(width=width, blocks=blocks, conv=conv), left_scale=left, right_scale=right), mlp=mlp)


def config(width, vocab, layers, positions=500, eps=1e-5):
    return dict(architecture="Ronavik", vocab=vocab, width=width, norm=dict(eps=eps), max_positions=positions, layers=layers)


# name -> config.json: both mixers, with and without a feed-forward; sizes that only the general kernels take (odd); values that are
# often equal or 1; more query heads a key head than a tile has rows, wide heads and values, many experts, long and short convolutions
CONFIGS = {
    "mixed": config(96, 200, [mamba2(mlp=moe(top=1)), parallel(mlp=moe(top=3)), parallel(heads=4, kv_heads=4, dim=16, vdim=64, width=96, blocks=2, conv=4, left=1.5, right=0.4, mlp=None),
                              mamba2(heads=4, vdim=32, state=16, groups=4, norm_groups=1, conv=2, mlp=None), mamba2(heads=2, vdim=48, state=48, groups=1, norm_groups=4, mlp=moe(5, 2, 32))]),
    "odd": config(60, 131, [parallel(3, 3, 9, 7, 0.3, 0.9, 3, 35, 5, 2, 1.1, 0.6, moe(5, 4, 11)), mamba2(3, 5, 7, 3, 3, 5, moe(3, 1, 13)), mamba2(5, 11, 33, 1, 6, 1, None), parallel(5, 1, 14, 21, 0.2, -0.3, 7, 18, 3, 5, 0.5, 0.9, moe(7, 7, 9))], 400, 1e-3),
    "ones": config(64, 96, [parallel(1, 1, 64, 64, 0.15, 1.0, 1, 64, 1, 1, 1.0, 1.0, moe(1, 1, 64)), mamba2(1, 64, 64, 1, 1, 1, moe(2, 1, 64)), mamba2(2, 32, 1, 1, 1, 1, None), parallel(2, 1, 8, 32, 0.5, 0.5, 500, 32, 32, 1, 1.0, 1.0, None)], 400, 1e-6),
    "wide": config(128, 320, [parallel(20, 1, 136, 200, 0.08, 0.5, 33, 256, 2, 6, 0.8, 1.0, moe(40, 8, 32)), mamba2(8, 64, 128, 2, 4, 8, moe(40, 20, 16)), parallel(16, 16, 24, 136, 0.2, 0.3, 64, 512, 16, 4, 1.0, 0.5, None)]),
}


def weights(cfg, seed=0):
    """{tensor name: float32 array of bf16 values} of a configuration."""
    rng, out = np.random.default_rng(seed), {}
    n = max([e["mlp"]["router"]["experts"] for e in cfg["layers"] if e["mlp"]], default=0)  # the columns that choose: 0 .. n - 1
    for name, shape in oracle.tensors(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            x = rng.normal(1, 0.2, shape)
            x[:n] = 1
        elif leaf in ("norm1b", "norm2b"):
            x = rng.normal(0.7, 0.2, shape)
            x[:n] = 0
        elif leaf == "norm":
            x = rng.normal(1.3, 0.3, shape)
        elif leaf == "conv":
            x = rng.normal(0, 0.7, shape)
        elif leaf == "lam":
            x = rng.normal(-3, 2, shape)
        elif leaf == "pb":
            x = rng.normal(-1.5, 0.7, shape)
        elif leaf == "D":
            x = rng.normal(0.8, 0.3, shape)
        elif leaf in ("dt_bias", "A_log"):
            x = rng.normal(-1.2, 0.8, shape)
        elif leaf == "b":
            x = rng.normal(0, 0.5, shape)
        elif name in ("embed", "pos"):
            x = rng.normal(0, 1.0 if name == "embed" else 0.5, shape)
            x[:, :n] = np.argsort(rng.random((shape[0], n)), axis=1) * (2.4 / n) - 1 if name == "embed" and n else 0
        elif leaf == "router":
            x = np.zeros(shape)
            x[:, n:] = rng.normal(0, 0.004 * shape[1] ** -0.5, (shape[0], shape[1] - n))
            x[np.arange(shape[0]), np.arange(shape[0])] = 2.5
        else:
            x = rng.normal(0, 1.3 * shape[-1] ** -0.5, shape)
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
