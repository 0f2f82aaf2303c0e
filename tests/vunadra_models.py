"""Small Vunadra configurations and checkpoints for the tests: random weights, made so that the parts that random weights would
hide are seen in the logits - attention that is peaked, convolutions that matter, a correction that forces one expert on every
token and keeps another from all - and so that no choice of experts is a close call: each token's embedding says in columns of
its own, which layers and passes leave in their order, how much it likes each expert."""
import numpy as np

from binutar_models import error, save  # noqa: F401  (a checkpoint is written, and logits are compared, as for the other design)
from oracle import vunadra as oracle


def dense(ff=64):
    return dict(kind="dense", ff=ff)


def moe(experts=6, identity=2, top=3, ff=48, limit=1.3, scale=1.7):
    return dict(kind="moe", router=dict(experts=experts, identity=identity, top=top, scale=scale), expert=dict(ff=ff, limit=limit))


def attention(heads=4, kv_heads=2, dim=24, vdim=40, conv=3, rot=24, base=500.0, scale=0.25, yarn=(3.0, 8.0, 64, 1.0), mlp=None):
    scaling = dict(zip(("factor", "fast", "original", "slow"), yarn))
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, scale=scale, rot=dict(base=base, dims=rot, scaling=scaling)), mlp=mlp)


def attention_2(heads=6, kv_heads=2, dim=16, size=20, rot=16, base=300.0, scale=0.3, softcap=4.0, waves=(3.0, 4.0, 1.0, 96), mlp=None):
    scaling = dict(zip(("factor", "high", "low", "original"), waves))
    return dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=size), scale=scale, softcap=softcap, rot=dict(base=base, dims=rot, scaling=scaling)), mlp=mlp)


def latent(heads=5, dim=16, rot_dim=8, vdim=24, rank=40, size=33, base=1000.0, scale=0.3, mlp=None):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, mask=dict(size=size), scale=scale, rot=dict(base=base, dims=rot_dim)), mlp=mlp)


def config(width, vocab, layers, loop=None, eps=1e-5, embed=0.7, logits=1.6):
    c = dict(architecture="Vunadra", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=embed), logit_scale=logits, layers=layers)
    return c | (dict(loop=dict(zip(("start", "stop", "times"), loop))) if loop else {})


# name -> config.json: a loop in the middle, all of the model as a loop, none; layers without a feed-forward; heads of which a part
# turns; sizes that only the general kernels take (odd); values that are often equal or 1; more query heads a key head than a tile
# has rows, wide heads, many experts; windows around the kernels' tiles
CONFIGS = {
    "mixed": config(96, 200, [attention(mlp=dense()), attention_2(mlp=moe()), latent(mlp=moe(top=2)), attention(conv=4, rot=10, mlp=None), attention_2(size=7, mlp=moe(identity=0))], (1, 4, 2)),
    "odd": config(60, 131, [attention(3, 1, 9, 7, 2, 6, mlp=dense(13)), attention_2(3, 3, 14, 5, 4, mlp=moe(5, 3, 4, 11)), latent(3, 11, 6, 9, 33, 17, mlp=dense(21))], (0, 3, 3), 1e-3, 1.3, 0.4),
    "ones": config(64, 96, [attention(1, 1, 64, 64, 1, 64, scale=0.15, mlp=moe(1, 1, 1, 64, 1.0, 1.0)), attention_2(1, 1, 64, 1, 64, scale=0.15, softcap=1.0, mlp=moe(1, 1, 2, 64)),
                            latent(1, 64, 64, 64, 64, 600, scale=0.1, mlp=dense(64))], (2, 3, 1), 1e-6, 1.0, 1.0),
    "wide": config(128, 320, [attention_2(20, 1, 136, 100, 72, scale=0.1, softcap=20.0, mlp=moe(40, 5, 8, 32)), attention(2, 1, 32, 16, 6, 32, mlp=moe(40, 1, 20, 16)), latent(24, 32, 16, 16, 128, 90, mlp=None)]),
    "windows": config(64, 128, [attention_2(4, 4, 32, n, 32, mlp=moe(4, 1, 2, 32)) for n in (64, 65, 16)] + [latent(4, 32, 32, 32, 64, n, mlp=None) for n in (48, 64)]),
}


def weights(cfg, seed=0):
    """{tensor name: float32 array of bf16 values} of a configuration."""
    rng, out, d = np.random.default_rng(seed), {}, cfg["width"]
    n = max([e["mlp"]["router"]["experts"] + e["mlp"]["router"]["identity"] for e in cfg["layers"] if e["mlp"] and e["mlp"]["kind"] == "moe"], default=0)  # the columns that choose: 0 .. n - 1
    for name, shape in oracle.tensors(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            x = rng.normal(1, 0.2, shape)
            x[:n] = 1
        elif leaf == "norm":
            x = rng.normal(1.2, 0.3, shape)
        elif leaf == "conv":
            x = rng.normal(0, 0.7, shape)
        elif leaf == "correction":
            x = np.zeros(shape)
            x[0], x[-1] = (1.5, 0) if shape[0] == 1 else (1.5, -1.5)
        elif leaf == "step":
            x = rng.normal(0, 0.6, shape)
            x[:, :n] = 0
        elif leaf == "b":
            x = rng.normal(0, 0.4, shape)
            if ".o." in name or ".down." in name:
                x[:n] = 0
        elif name == "embed":
            x = rng.normal(0, 1.0, shape)
            x[:, :n] = np.argsort(rng.random((shape[0], n)), axis=1) * (2.0 / n) if n else x[:, :n]
        elif name == "loop.in":
            x = rng.normal(0, 0.8 * shape[1] ** -0.5, shape)
            x[:n] = 0
            x[np.arange(n), d + np.arange(n)] = 1
        elif leaf == "router":
            x = np.zeros(shape)
            x[:, n:] = rng.normal(0, 0.004 * d ** -0.5, (shape[0], d - n))
            x[np.arange(shape[0]), np.arange(shape[0])] = 2.5
        else:
            x = rng.normal(0, (0.6 if leaf == "down" else 1.3) * shape[1] ** -0.5, shape)
            if leaf in ("o", "down"):
                x[:n] = 0
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
