"""Typed configuration of the Soporax decoder: a list of layers, each with a mixer and a feed-forward of its own, and a group
of neighbouring layers that runs several times.

config.json::

    {"architecture": "Soporax", "vocab": V, "width": W, "norm": {"eps": e}, "logit_scale": a,
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [
       {"type": "attention",
        "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s, "mask": {"size": w}},
        "mlp": {"kind": "dense", "ff": f, "limit": l}},
       {"type": "attention_2",
        "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s,
                  "rot": {"base": b, "dims": n, "scaling": {"factor": c, "low": l, "high": h, "original": o}}},
        "mlp": {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "top": k}}},
       {"type": "latent_attention",
        "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "q_rank": q, "kv_rank": k, "scale": s,
                  "rot": {"base": b, "dims": r, "scaling": {"factor": c, "original": o, "fast": f, "slow": l}}},
        "mlp": null},
       ...]}

``mlp`` null means the layer has no feed-forward; ``loop`` absent or null means every layer runs once; ``mask`` absent means
no window, ``rot`` no rotation, ``scaling`` plain frequencies.  Every size and constant is read from here; a key that is
absent, of the wrong type or out of range is an error that names it.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .fields import ConfigError, KeyReader

MIXER_TYPES = ("attention", "attention_2", "latent_attention")
MLP_KINDS = ("dense", "moe")


@dataclass
class SoporaxLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


def _rotation(r: KeyReader, where: str, most: int, scaling_keys) -> Optional[Dict[str, Any]]:
    if not r.has("rot"):
        return None
    t = KeyReader(r.raw("rot"), where + ".rot")
    out: Dict[str, Any] = {"base": t.number("base", positive=True), "dims": t.integer("dims", minimum=0), "scaling": None}
    if out["dims"] % 2 != 0 or out["dims"] > most:
        raise ConfigError(f"{where}.rot: dims {out['dims']} must be even and at most {most}")
    if t.has("scaling"):
        s = KeyReader(t.raw("scaling"), where + ".rot.scaling")
        out["scaling"] = {k: s.number(k, positive=True) for k in scaling_keys}
    return out


def _attention(obj: Any, where: str, kind: str) -> Dict[str, Any]:
    r = KeyReader(obj, where)
    out: Dict[str, Any] = {"heads": r.integer("heads", minimum=1), "kv_heads": r.integer("kv_heads", minimum=1),
                           "dim": r.integer("dim", minimum=1), "vdim": r.integer("vdim", minimum=1),
                           "scale": r.number("scale", positive=True)}
    if out["heads"] % out["kv_heads"] != 0:
        raise ConfigError(f"{where}: {out['heads']} heads cannot share {out['kv_heads']} kv_heads")
    if kind == "attention":
        out["mask"] = None
        if r.has("mask"):
            out["mask"] = {"size": KeyReader(r.raw("mask"), where + ".mask").integer("size", minimum=1)}
    else:
        out["rot"] = _rotation(r, where, out["dim"], ("factor", "low", "high", "original"))
    return out


def _latent(obj: Any, where: str) -> Dict[str, Any]:
    r = KeyReader(obj, where)
    out: Dict[str, Any] = {k: r.integer(k, minimum=1) for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
    out["rot_dim"] = r.integer("rot_dim", minimum=0)
    out["scale"] = r.number("scale", positive=True)
    out["rot"] = _rotation(r, where, out["rot_dim"], ("factor", "original", "fast", "slow"))
    return out


def _mlp(obj: Any, where: str) -> Dict[str, Any]:
    m = KeyReader(obj, where)
    kind = m.string("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"{where}: kind {kind!r} is not one of {MLP_KINDS}")
    if kind == "dense":
        return {"kind": kind, "ff": m.integer("ff", minimum=1), "limit": m.number("limit", positive=True)}
    r = KeyReader(m.raw("router"), where + ".router")
    router = {"experts": r.integer("experts", minimum=1), "top": r.integer("top", minimum=1)}
    if router["top"] > router["experts"]:
        raise ConfigError(f"{where}.router: top {router['top']} exceeds the {router['experts']} experts")
    return {"kind": kind, "expert": {"ff": KeyReader(m.raw("expert"), where + ".expert").integer("ff", minimum=1)},
            "router": router}


@dataclass
class SoporaxConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    loop: Optional[Dict[str, int]] = None
    layers: List[SoporaxLayer] = field(default_factory=list)
    architecture: str = "Soporax"

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("config.json: 'vocab' and 'width' must be >= 1")
        if not self.norm_eps > 0:
            raise ConfigError("config.json: key 'norm.eps' must be > 0")
        if not self.layers:
            raise ConfigError("config.json: key 'layers' must list at least one layer")
        if self.loop is not None:
            start, stop, times = (self.loop[k] for k in ("start", "stop", "times"))
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ConfigError(f"config.json: loop: layers {start} .. {stop - 1} of {len(self.layers)}, {times} times, "
                                  "are not a group of layers that runs at least once")

    @classmethod
    def from_dict(cls, obj: Dict[str, Any]) -> "SoporaxConfig":
        r = KeyReader(obj)
        norm = KeyReader(r.raw("norm"), "config.json: norm")
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list):
            raise ConfigError("config.json: key 'layers' must be a list")
        layers = []
        for i, entry in enumerate(raw_layers):
            where = f"config.json: layers[{i}]"
            e = KeyReader(entry, where)
            kind = e.string("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}: type {kind!r} is not one of {MIXER_TYPES}")
            mixer = e.raw("mixer")
            mixer = _latent(mixer, where + ".mixer") if kind == "latent_attention" else _attention(mixer, where + ".mixer", kind)
            layers.append(SoporaxLayer(kind, mixer, _mlp(e.raw("mlp"), where + ".mlp") if e.has("mlp") else None))
        loop = None
        if r.has("loop"):
            t = KeyReader(r.raw("loop"), "config.json: loop")
            loop = {k: t.integer(k, minimum=low) for k, low in (("start", 0), ("stop", 1), ("times", 1))}
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=norm.number("eps", positive=True), logit_scale=r.number("logit_scale", 1.0), loop=loop,
                   layers=layers, architecture=r.string("architecture", "Soporax"))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "loop": copy.deepcopy(self.loop),
                "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)}
                           for l in self.layers]}
