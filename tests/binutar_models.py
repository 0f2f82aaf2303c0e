"""Small Binutar configurations and checkpoints for the tests: random weights, scaled so that the parts that random weights
would hide are seen in the logits - attention that is peaked and reaches far, sinks that matter, states that last."""
import json
import os
import struct

import numpy as np

from oracle import binutar as oracle


def latent(heads=4, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=56, scaling=True, base=3000.0, scale=0.7, ff=96, limit=1.6):
    rot = dict(base=base, dims=rot_dim) | (dict(scaling=dict(factor=2.5, original=256, fast=20.0, slow=1.5)) if scaling else {})
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, rot=rot, scale=scale),
                mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None)


def lightning(heads=3, dim=16, vdim=24, decay=(0.35, 0.93, 0.998), ff=80, limit=0.9):
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay)), mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None)


# name -> config.json: both mixers in turn; sizes that only the general kernels take (odd, no multiple of 8); values that are
# often equal or 1 (heads of one, a latent as wide as the model); layers without a feed-forward, one kind of mixer alone
CONFIGS = {
    "turns": dict(architecture="Binutar", vocab=200, width=96, norm=dict(eps=1e-5), layers=[latent(), lightning(), latent(heads=2, rot_dim=8, scaling=False, ff=64), lightning(dim=32)]),
    "odd": dict(architecture="Binutar", vocab=131, width=60, norm=dict(eps=1e-3),
                layers=[lightning(heads=2, dim=9, vdim=7, decay=(0.5, 0.99), ff=33), latent(heads=3, dim=10, rot_dim=6, vdim=11, kv_rank=19, q_rank=13, ff=21)]),
    "ones": dict(architecture="Binutar", vocab=96, width=64, norm=dict(eps=1e-6), layers=[latent(heads=1, dim=64, rot_dim=2, vdim=64, kv_rank=64, q_rank=64, ff=None), lightning(heads=1, decay=(1.0,), ff=None)]),
    "wide": dict(architecture="Binutar", vocab=320, width=128, norm=dict(eps=1e-5), layers=[latent(heads=20, dim=32, rot_dim=32, vdim=16, kv_rank=256, q_rank=72, ff=160), lightning(heads=2, dim=128, vdim=64, decay=(0.8, 0.995))]),
    "linear": dict(architecture="Binutar", vocab=128, width=64, norm=dict(eps=1e-5), layers=[lightning(heads=3, dim=48), lightning(heads=2, dim=64, vdim=32, decay=(0.6, 0.99))]),
}


def weights(cfg, seed=0):
    """{tensor name: float32 array of bf16 values} of a configuration."""
    rng, out = np.random.default_rng(seed), {}
    for name, shape in oracle.tensors(cfg).items():
        if name.endswith(".alpha"):
            x = rng.uniform(0.4, 0.9, shape)
        elif name.endswith("sink"):
            x = rng.normal(1.0, 1.5, shape)
        elif len(shape) == 1:
            x = rng.normal(0.0, 0.2, shape) if name.endswith(".b") else rng.normal(1.0, 0.25, shape)
        elif name == "embed":
            x = rng.normal(0, 1.0, shape)
        else:
            x = rng.normal(0, 1.3 * shape[1] ** -0.5, shape)
        bits = np.asarray(x, np.float32).reshape(-1).view(np.uint32)
        bits = ((bits + (0x7FFF + (bits >> 16 & 1))) >> 16 << 16).astype(np.uint32)
        out[name] = bits.view(np.float32).reshape(shape)
    return out


def save(folder, cfg, w):
    """config.json and model.safetensors (BF16) of a configuration and its weights."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, x in w.items():
        raw = (np.ascontiguousarray(x, np.float32).reshape(-1).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(x)), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return str(folder)


class Alone:
    """The oracle's logits of one token sequence, with what it needs kept between calls."""

    def __init__(self, cfg, w):
        self.cfg, self.w, self.caches, self.at = cfg, w, oracle.caches(cfg), 0

    def __call__(self, ids):
        out = oracle.forward(ids, self.at, self.w, self.cfg, self.caches)
        self.at += len(ids)
        return out


def greedy(cfg, w, prompt, n):
    """(tokens, least distance between the best two logits) of a greedy continuation."""
    run, made, margin = Alone(cfg, w), [], np.inf
    out = run(prompt)
    for _ in range(n):
        top = np.sort(out[-1])[-2:]
        margin = min(margin, top[1] - top[0])
        made.append(int(out[-1].argmax()))
        out = run(made[-1:])
    return made, margin


def error(got, want):
    """The largest root mean square difference of a row of logits, over the logits' own."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return float((np.sqrt((d ** 2).mean(-1)) / want.std()).max())
