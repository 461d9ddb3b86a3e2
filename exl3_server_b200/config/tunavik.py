"""Typed configuration of the Tunavik decoder: a list of attention layers, each with sizes and a routed feed-forward of its
own.

config.json::

    {"architecture": "Tunavik", "vocab": V, "width": W, "norm": {"eps": e}, "logit_scale": a, "logit_softcap": c,
     "layers": [
       {"type": "attention",
        "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s, "bias_max": D,
                  "q_temp": {"coef": a, "every": n}, "kv_from": j},
        "mlp": {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "top": k}, "shared": {"ff": f}}},
       ...]}

``mlp`` null means the layer has no feed-forward; ``kv_from``, ``q_temp``, ``shared`` and ``logit_softcap`` absent or null
mean the thing is not there.  ``kv_from`` names the earlier layer whose keys and values the layer reads.  Every size and
constant is read from here (the length of a layer's distance table is the checkpoint's); a key that is absent, of the wrong
type or out of range is an error that names it.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .fields import ConfigError, KeyReader

MIXER_TYPES = ("attention",)
MLP_KINDS = ("moe",)


@dataclass
class TunavikLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


def _attention(obj: Any, where: str) -> Dict[str, Any]:
    r = KeyReader(obj, where)
    out: Dict[str, Any] = {"heads": r.integer("heads", minimum=1), "kv_heads": r.integer("kv_heads", minimum=1),
                           "dim": r.integer("dim", minimum=1), "vdim": r.integer("vdim", minimum=1),
                           "scale": r.number("scale", positive=True), "bias_max": r.number("bias_max", positive=True)}
    if out["bias_max"] == int(out["bias_max"]):
        out["bias_max"] = int(out["bias_max"])
    if out["heads"] % out["kv_heads"] != 0:
        raise ConfigError(f"{where}: {out['heads']} heads cannot share {out['kv_heads']} kv_heads")
    out["q_temp"] = None
    if r.has("q_temp"):
        t = KeyReader(r.raw("q_temp"), where + ".q_temp")
        out["q_temp"] = {"coef": t.number("coef"), "every": t.number("every", positive=True)}
    out["kv_from"] = r.integer("kv_from", minimum=0) if r.has("kv_from") else None
    return out


def _mlp(obj: Any, where: str) -> Dict[str, Any]:
    m = KeyReader(obj, where)
    kind = m.string("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"{where}: kind {kind!r} is not one of {MLP_KINDS}")
    ff = lambda key: {"ff": KeyReader(m.raw(key), f"{where}.{key}").integer("ff", minimum=1)}
    r = KeyReader(m.raw("router"), where + ".router")
    router = {"experts": r.integer("experts", minimum=1), "top": r.integer("top", minimum=1)}
    if router["top"] > router["experts"]:
        raise ConfigError(f"{where}.router: top {router['top']} exceeds the {router['experts']} experts")
    return {"kind": kind, "expert": ff("expert"), "router": router, "shared": ff("shared") if m.has("shared") else None}


@dataclass
class TunavikConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    logit_softcap: Optional[float]
    layers: List[TunavikLayer] = field(default_factory=list)
    architecture: str = "Tunavik"

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("config.json: 'vocab' and 'width' must be >= 1")
        if not self.norm_eps > 0:
            raise ConfigError("config.json: key 'norm.eps' must be > 0")
        if self.logit_scale == 0:
            raise ConfigError("config.json: key 'logit_scale' must not be 0")
        if not self.layers:
            raise ConfigError("config.json: key 'layers' must list at least one layer")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            j = m.get("kv_from")
            if j is None:
                continue
            where = f"config.json: layers[{i}].mixer"
            if not 0 <= j < i:
                raise ConfigError(f"{where}: kv_from {j} is not an earlier layer")
            src = self.layers[j].mixer
            if src.get("kv_from") is not None:
                raise ConfigError(f"{where}: kv_from {j} has no keys and values of its own")
            if any(m[k] != src[k] for k in ("kv_heads", "dim", "vdim")):
                raise ConfigError(f"{where}: kv_heads, dim and vdim must be those of layer {j}, whose keys and values it reads")

    @classmethod
    def from_dict(cls, obj: Dict[str, Any]) -> "TunavikConfig":
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
            mlp = _mlp(e.raw("mlp"), where + ".mlp") if e.has("mlp") else None
            layers.append(TunavikLayer(kind, _attention(e.raw("mixer"), where + ".mixer"), mlp))
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=norm.number("eps", positive=True), logit_scale=r.number("logit_scale", 1.0),
                   logit_softcap=r.number("logit_softcap", positive=True) if r.has("logit_softcap") else None,
                   layers=layers, architecture=r.string("architecture", "Tunavik"))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
                "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)}
                           for l in self.layers]}
