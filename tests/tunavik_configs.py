"""Small Tunavik configurations for the tests, different in every size and option, with random weights."""
from __future__ import annotations

import os

import torch
from safetensors import safe_open

from exl3_server_b200 import write_random_model
from exl3_server_b200.config.tunavik import TunavikConfig, TunavikLayer
from exl3_server_b200.weights.safetensors_io import write_safetensors


def attn(heads, kv_heads, dim, vdim, scale, bias_max, temp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def L(mixer, mlp=None):
    return TunavikLayer("attention", mixer, mlp)


def cfg(vocab, width, eps, logit_scale, softcap, layers):
    return TunavikConfig(vocab=vocab, width=width, norm_eps=eps, logit_scale=logit_scale, logit_softcap=softcap, layers=layers)


CONFIGS = {
    # layers that read the keys and values of the layer before, of one further back (with other heads of their own, another
    # scale, table and temperature) and of the same one as another reader; values narrower and wider than keys; layers
    # without a feed-forward, without a shared expert, without a temperature, one pick, every expert picked
    "mixed": cfg(211, 96, 1e-5, 1.7, 3.0, [
        L(attn(4, 2, 24, 16, 0.21, 50, (0.5, 10)), moe(40, 9, 3, shared=56)),
        L(attn(6, 3, 16, 40, 0.25, 21, (0.2, 1))),
        L(attn(8, 2, 24, 16, 0.15, 300, (-0.1, 33), kv_from=0), moe(24, 5, 1)),
        L(attn(3, 3, 16, 40, 0.3, 97, kv_from=1), moe(48, 4, 4, shared=20)),
        L(attn(2, 2, 24, 16, 0.2, 64, (0.3, 64), kv_from=0)),
        L(attn(4, 4, 32, 32, 0.17, 160, (0.25, 7)), moe(32, 6, 2, shared=32)),
    ]),
    # sizes that are multiples of nothing, an odd width, one expert, no soft cap
    "odd": cfg(97, 101, 1e-6, 0.6, None, [
        L(attn(3, 3, 10, 6, 0.4, 30, (0.7, 3)), moe(12, 1, 1, shared=20)),
        L(attn(5, 1, 14, 22, 0.3, 40, (0.1, 100)), moe(30, 7, 2)),
        L(attn(3, 3, 10, 6, 0.3, 200, (0.2, 5), kv_from=0), moe(18, 3, 3, shared=10)),
        L(attn(2, 1, 9, 33, 0.35, 26), None),
    ]),
    # heads of 64 and 128 features (the tensor-core kernels' own rows) and narrower ones that are kept in such rows, more
    # query heads on a key/value head than the decode kernel takes, widths for the experts' tensor-core product
    "wide": cfg(301, 128, 1e-5, 2.5, 12.0, [
        L(attn(4, 2, 64, 64, 0.11, 90, (0.3, 20)), moe(64, 8, 2, shared=64)),
        L(attn(4, 1, 128, 128, 0.08, 400, (0.1, 50)), None),
        L(attn(16, 1, 40, 72, 0.14, 33), moe(72, 5, 3, shared=40)),
        L(attn(20, 1, 16, 16, 0.22, 128, (0.4, 30)), moe(40, 4, 1)),
        L(attn(2, 2, 64, 64, 0.1, 48, (0.2, 11), kv_from=0), None),
        L(attn(2, 1, 160, 136, 0.07, 70, (0.1, 9)), moe(64, 6, 2)),
    ]),
    # each mechanism alone
    "only_attention": cfg(128, 64, 1e-5, 1.5, None, [L(attn(4, 2, 32, 16, 0.4, 80, (0.2, 40)))]),
    "only_tiles": cfg(128, 64, 1e-5, 1.5, None, [L(attn(4, 1, 64, 64, 0.3, 80))]),
    "only_reader": cfg(128, 64, 1e-5, 1.0, 9.0, [L(attn(2, 2, 32, 32, 0.3, 60)), L(attn(6, 2, 32, 32, 0.2, 45, (0.5, 25), kv_from=0))]),
    "only_moe": cfg(128, 64, 1e-5, 1.2, 5.0, [L(attn(1, 1, 8, 8, 0.3, 24), moe(24, 14, 3, shared=16))]),
}


def random_config(seed: int) -> TunavikConfig:
    """A configuration drawn from a seed: two to five layers, every size, count and constant drawn anew, any later layer
    reading an earlier one's keys and values, a routed or no feed-forward beside each."""
    import random
    r = random.Random(seed)
    width = r.choice([48, 72, 80, 104, 136])
    layers = []
    for i in range(r.randint(2, 5)):
        owners = [j for j in range(i) if layers[j].mixer.get("kv_from") is None]
        src = r.choice(owners) if owners and r.random() < 0.4 else None
        if src is None:
            kv, dim, vdim = r.randint(1, 3), r.choice([6, 8, 16, 24, 32, 64]), r.choice([8, 12, 16, 32, 64])
        else:
            kv, dim, vdim = (layers[src].mixer[k] for k in ("kv_heads", "dim", "vdim"))
        temp = (r.uniform(0.05, 0.5), r.choice([1, 3, 16, 100, 4096])) if r.random() < 0.8 else None
        mixer = attn(kv * r.randint(1, 5), kv, dim, vdim, r.uniform(0.1, 0.4), r.choice([25, 36, 64, 250, 1000]), temp, src)
        experts = r.randint(1, 10)
        mlp = None if r.random() < 0.25 else moe(r.choice([8, 24, 40]), experts, r.randint(1, min(4, experts)),
                                                 shared=r.choice([None, 16, 40]))
        layers.append(L(mixer, mlp))
    return cfg(r.randint(40, 300), width, r.choice([1e-6, 1e-5, 1e-4]), r.uniform(0.5, 4.0),
               r.choice([None, 4.0, 20.0, 50.0]), layers)


RANDOM_SEEDS = list(range(300, 310))
CONFIGS.update({f"random{seed}": random_config(seed) for seed in RANDOM_SEEDS})

ROUTED = {name for name, c in CONFIGS.items() if any(l.mlp for l in c.layers)}


def table_rows(i: int, bias_max: float) -> int:
    """Rows of layer i's distance table: of every kind of length, odd ones and the shortest too."""
    rows = (16, 9, 40, 2, 26, 6)[i % 6]
    while rows // 2 >= bias_max:
        rows -= 8
    return rows


def make_tunavik(name: str, folder: str, std: float = 0.06) -> str:
    """std 0.06, and what random weights of that size would hide drawn otherwise: distance tables of +-2 (a wrong row shows),
    sinks of -1 .. 2 (a sink left out changes every row), biases of the projections and of the router of some tenths, larger
    routers, norm weights spread around what they are stored around."""
    write_random_model(CONFIGS[name], folder, seed=2311 + sum(map(ord, name)), std=std, norm_std=0.2, dtype=torch.bfloat16)
    path = os.path.join(folder, "model.safetensors")
    with safe_open(path, framework="pt") as f:
        tensors = {k: f.get_tensor(k) for k in f.keys()}
    g = torch.Generator().manual_seed(13)
    rnd = lambda shape: torch.rand(shape, generator=g)
    layers = CONFIGS[name].layers
    for k in sorted(tensors):
        t = tensors[k]
        last = k.rsplit(".", 1)[-1]
        if last == "rel":
            i = int(k[1:k.index(".")])
            tensors[k] = ((rnd((table_rows(i, layers[i].mixer["bias_max"]), t.shape[1])) - 0.5) * 4.0).to(torch.bfloat16)
        elif last == "sink":
            tensors[k] = (3.0 * rnd(t.shape) - 1.0).to(torch.bfloat16)
        elif k.endswith(".mlp.router"):
            tensors[k] = (t.float() * 3.0).to(torch.bfloat16)
        elif last == "b":
            tensors[k] = ((rnd(t.shape) - 0.5) * 0.6).to(torch.bfloat16)
        elif last in ("norm1", "norm2") or k in ("embed.norm", "final.norm"):
            tensors[k] = ((rnd(t.shape) - 0.5) * 0.6).to(torch.bfloat16)
    write_safetensors(path, tensors.items(), metadata={"format": "pt"})
    return folder
