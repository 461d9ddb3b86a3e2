"""Small Soporax configurations for the tests, different in every size and option, with random weights."""
from __future__ import annotations

import os

import torch
from safetensors import safe_open

from exl3_server_b200 import write_random_model
from exl3_server_b200.config.soporax import SoporaxConfig, SoporaxLayer
from exl3_server_b200.weights.safetensors_io import write_safetensors


def bands(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def ramp(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def window(heads, kv_heads, dim, vdim, scale, size):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}


def rotated(heads, kv_heads, dim, vdim, scale, dims, base=10000.0, scaling=None):
    return "attention_2", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                           "rot": {"base": base, "dims": dims, "scaling": scaling}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, scaling=None):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                "kv_rank": kv_rank, "scale": scale,
                                "rot": {"base": base, "dims": rot_dim, "scaling": scaling}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def L(mixer, mlp=None):
    return SoporaxLayer(mixer[0], mixer[1], mlp)


def cfg(vocab, width, eps, logit_scale, layers, loop=None):
    keys = ("start", "stop", "times")
    return SoporaxConfig(vocab=vocab, width=width, norm_eps=eps, logit_scale=logit_scale, layers=layers,
                         loop=dict(zip(keys, loop)) if loop else None)


CONFIGS = {
    # every mixer and feed-forward, two layers in the middle that run four times; values narrower and wider than keys; two and
    # three picks; a layer without a feed-forward; frequencies of every band
    "mixed": cfg(211, 96, 1e-5, 1.7, [
        L(rotated(6, 3, 24, 16, 0.21, 16, 500.0, bands(4.0, 1.0, 4.0, 40)), moe(40, 9, 2)),
        L(latent(5, 24, 16, 40, 44, 56, 0.15, 3000.0, ramp(6.0, 64, 8.0, 1.0)), dense(72, 0.6)),
        L(window(4, 2, 16, 40, 0.5, 37), moe(24, 5, 3)),
        L(latent(3, 16, 8, 16, 20, 32, 0.2), moe(32, 6, 1)),
        L(window(6, 1, 32, 24, 0.3, 64)),
        L(rotated(8, 2, 16, 32, 0.25, 16, 10000.0, bands(8.0, 2.0, 3.0, 100)), dense(40, 2.5)),
    ], loop=(1, 3, 4)),
    # sizes that are multiples of nothing, an odd width; the loop begins with the first layer; one expert, every expert picked
    "odd": cfg(97, 101, 1e-6, 0.6, [
        L(window(3, 3, 10, 6, 0.9, 1), moe(12, 1, 1)),
        L(rotated(5, 1, 14, 22, 0.3, 6, 100.0), moe(30, 3, 3)),
        L(latent(3, 9, 6, 13, 17, 21, 0.3, 50.0, ramp(3.0, 30, 4.0, 0.5)), dense(50, 1.0)),
        L(rotated(2, 1, 9, 33, 0.35, 0), None),
    ], loop=(0, 2, 3)),
    # heads of 64 and 128 features and narrower ones in such rows, more query heads on a key/value head than the decode kernel
    # takes, widths for the experts' tensor-core product, the loop is the last layer alone
    "wide": cfg(301, 128, 1e-5, 2.5, [
        L(rotated(4, 2, 64, 64, 0.11, 64, 10000.0, bands(2.0, 1.0, 4.0, 128)), moe(64, 8, 2)),
        L(window(4, 1, 128, 128, 0.2, 150), moe(72, 5, 3)),
        L(window(20, 1, 16, 48, 0.4, 65), None),
        L(rotated(2, 1, 160, 136, 0.07, 32), dense(96, 3.0)),
        L(latent(7, 48, 32, 64, 80, 112, 0.1, 10000.0, ramp(4.0, 128, 16.0, 2.0)), moe(40, 4, 1)),
        L(window(16, 1, 64, 64, 0.3, 100), moe(64, 6, 4)),
    ], loop=(5, 6, 3)),
    # the whole model runs twice, and a model without a loop
    "twice": cfg(128, 64, 1e-5, 1.1, [L(rotated(4, 1, 32, 16, 0.2, 8), dense(40, 0.8)), L(window(2, 2, 16, 16, 0.6, 20))], loop=(0, 2, 2)),
    "once": cfg(128, 72, 1e-5, 1.0, [L(latent(4, 16, 8, 24, 40, 48, 0.2), moe(24, 7, 2)), L(rotated(4, 4, 24, 24, 0.2, 24), moe(16, 3, 1))]),
    # each mechanism alone
    "only_window": cfg(128, 64, 1e-5, 1.5, [L(window(4, 2, 32, 16, 0.4, 50))]),
    "only_window_tiles": cfg(128, 64, 1e-5, 1.5, [L(window(4, 1, 64, 64, 0.3, 200))]),
    "only_rotated": cfg(128, 64, 1e-5, 1.5, [L(rotated(4, 2, 40, 24, 0.3, 8, 10000.0, bands(8.0, 1.0, 4.0, 64)))]),
    "only_rotated_tiles": cfg(128, 64, 1e-5, 1.5, [L(rotated(4, 2, 64, 64, 0.2, 32, 10000.0, bands(8.0, 1.0, 4.0, 64)))]),
    "only_latent": cfg(128, 64, 1e-5, 1.5, [L(latent(4, 32, 16, 24, 40, 48, 0.2, 10000.0, ramp(4.0, 64, 8.0, 1.0)))]),
    "only_moe": cfg(128, 64, 1e-5, 1.2, [L(window(1, 1, 8, 8, 0.3, 1), moe(24, 14, 3))]),
    "only_dense": cfg(128, 64, 1e-5, 1.2, [L(window(1, 1, 8, 8, 0.3, 1), dense(48, 0.4))]),
}


def random_config(seed: int) -> SoporaxConfig:
    """A configuration drawn from a seed: two to five layers, every size, count and constant drawn anew, a loop over any group
    of them or none."""
    import random
    r = random.Random(seed)
    width = r.choice([48, 72, 80, 104, 136])
    layers = []
    for _ in range(r.randint(2, 5)):
        kv, dim, vdim = r.randint(1, 3), r.choice([6, 8, 16, 24, 32, 64, 128]), r.choice([8, 12, 16, 32, 64])
        heads, base = kv * r.randint(1, 5), r.choice([50.0, 10000.0, 500000.0])
        kind = r.randrange(3)
        if kind == 0:
            mixer = window(heads, kv, dim, vdim, r.uniform(0.2, 0.6), r.choice([1, 2, 17, 63, 64, 65, 100, 1000]))
        elif kind == 1:
            scaling = bands(r.choice([2.0, 8.0]), 1.0, r.choice([2.0, 4.0]), r.choice([32, 200])) if r.random() < 0.8 else None
            mixer = rotated(heads, kv, dim, vdim, r.uniform(0.1, 0.4), r.randrange(0, dim // 2 + 1) * 2, base, scaling)
        else:
            scaling = ramp(r.choice([1.5, 4.0, 16.0]), r.choice([32, 200]), r.choice([4.0, 16.0]), r.choice([0.5, 1.0])) \
                if r.random() < 0.8 else None
            mixer = latent(r.randint(1, 6), dim, r.choice([2, 8, 16, 32]), vdim, r.choice([12, 40, 64]), r.choice([16, 24, 48, 96]),
                           r.uniform(0.1, 0.3), base, scaling)
        experts = r.randint(1, 10)
        mlp = r.choice([None, dense(r.choice([24, 56]), r.choice([0.3, 1.0, 5.0])), moe(r.choice([8, 24, 40]), experts, r.randint(1, min(4, experts))),
                        moe(r.choice([8, 24, 40]), experts, 1)])
        layers.append(L(mixer, mlp))
    loop = None
    if r.random() < 0.8:
        start = r.randrange(len(layers))
        loop = (start, r.randint(start + 1, len(layers)), r.randint(1, 3))
    return cfg(r.randint(40, 300), width, r.choice([1e-6, 1e-5, 1e-4]), r.uniform(0.5, 4.0), layers, loop)


RANDOM_SEEDS = list(range(500, 512))
CONFIGS.update({f"random{seed}": random_config(seed) for seed in RANDOM_SEEDS})


def make_soporax(name: str, folder: str, std: float = 0.06) -> str:
    """std 0.06, and what random weights of that size would hide drawn otherwise: sinks of -1 .. 2, biases of some tenths,
    gates and the bounded gate's two projections several times larger (so that bounds and gates act), a pass's vector of the
    embedding's size, norm weights spread around one."""
    write_random_model(CONFIGS[name], folder, seed=4177 + sum(map(ord, name)), std=std, norm_std=0.2, dtype=torch.bfloat16)
    path = os.path.join(folder, "model.safetensors")
    with safe_open(path, framework="pt") as f:
        tensors = {k: f.get_tensor(k) for k in f.keys()}
    g = torch.Generator().manual_seed(17)
    rnd = lambda shape: torch.rand(shape, generator=g)
    for k in sorted(tensors):
        t = tensors[k]
        last = k.rsplit(".", 1)[-1]
        if last == "sink":
            tensors[k] = (3.0 * rnd(t.shape) - 1.0).to(torch.bfloat16)
        elif last == "b":
            tensors[k] = ((rnd(t.shape) - 0.5) * 0.6).to(torch.bfloat16)
        elif last == "g" or k.endswith(".mlp.gate") or k.endswith(".mlp.up"):
            tensors[k] = (t.float() * 4.0).to(torch.bfloat16)
        elif last == "step":
            tensors[k] = ((rnd(t.shape) - 0.5) * 0.3).to(torch.bfloat16)
    write_safetensors(path, tensors.items(), metadata={"format": "pt"})
    return folder
