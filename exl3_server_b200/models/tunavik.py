"""The Tunavik decoder as a plan of parts.

The embedding is the token's row plus a sinusoidal vector of its position, normed (``table_sinusoid``).  Every layer norms
its sublayers' outputs only (``outnorm``), with norm weights stored around zero.  Layers come from the configuration's list:

* ``attention``: grouped-query attention with biases on all four projections, one norm over all query heads and one over
  all key heads, a query temperature that grows with the position, a learned bias of the scores by distance and a learned
  sink per head; no rotation (``normed_attention`` with these options).  A layer with ``kv_from`` has queries only and reads
  the named layer's cache through its schedule entry;
* feed-forwards are routed (``routed``: biased logits, the softmax over the picks alone, squared-relu experts, an ungated
  shared expert), or absent.

The last norm's output times a constant goes to an untied head whose logits may be soft-capped.

Tensor names: ``embed``, ``embed.norm``, ``final.norm``, ``head`` and, per layer ``l<i>``: ``norm1``, ``norm2``, ``mix.*`` and
``mlp.*`` (see the parts' modules).
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tunavik import TunavikConfig
from ..parts.spec import (EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerSpec, MixerSpec, ModelPlan, NormSpec,
                          ScheduleEntry)

NAMES = ("Tunavik", "tunavik")
SINUSOID_BASE = 10000.0


def _norm(cfg: TunavikConfig) -> NormSpec:
    return NormSpec(kind="rms", width=cfg.width, eps=cfg.norm_eps, params={"suffix": "", "one_plus": True})


def _attention(cfg: TunavikConfig, m: dict) -> MixerSpec:
    temp = m.get("q_temp")
    return MixerSpec(kind="normed_attention", width=cfg.width, heads=m["heads"], kv_heads=m["kv_heads"],
                     head_dim=m["dim"], softmax_scale=m["scale"], position=None,
                     params={"value_dim": m["vdim"], "bias": True, "qk_norm": "rows", "norm_eps": cfg.norm_eps,
                             "sink": "learned", "distance_bias": m["bias_max"],
                             "q_temp": (temp["coef"], temp["every"]) if temp else None,
                             "reads_kv": m.get("kv_from") is not None, "tile_rows": True})


def _feed_forward(cfg: TunavikConfig, mlp: dict) -> FeedForwardSpec:
    return FeedForwardSpec(kind="routed", width=cfg.width, inner=mlp["expert"]["ff"],
                           params={"experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "score": "picked",
                                   "correction": False, "router_bias": True, "activation": "relu2", "shared_gate": False,
                                   "shared_inner": mlp["shared"]["ff"] if mlp.get("shared") else 0})


def build_plan(cfg: TunavikConfig) -> ModelPlan:
    layers, schedule, ignorable = [], [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ff = _feed_forward(cfg, layer.mlp) if layer.mlp is not None else None
        if ff is None:
            ignorable.append(p + "norm2")                        # nothing reads it in a layer without a feed-forward
        layers.append(LayerSpec(
            arrangement="outnorm", mixer=_attention(cfg, layer.mixer), feed_forward=ff, mixer_norm=_norm(cfg),
            feed_forward_norm=_norm(cfg) if ff is not None else None, residual_scale=1.0,
            names={"mixer": p + "mix.", "feed_forward": p + "mlp.", "mixer_norm": p + "norm1",
                   "feed_forward_norm": p + "norm2"}))
        schedule.append(ScheduleEntry(layer=i, cache_from=layer.mixer.get("kv_from")))
    plan = ModelPlan(
        architecture=cfg.architecture,
        embedding=EmbeddingSpec(vocab=cfg.vocab, width=cfg.width, scale=1.0, name="embed", kind="table_sinusoid",
                                params={"base": SINUSOID_BASE, "norm": _norm(cfg), "norm_name": "embed.norm"}),
        layers=layers, schedule=schedule, final_norm=_norm(cfg), final_norm_name="final.norm",
        head=HeadSpec(vocab=cfg.vocab, width=cfg.width, input_divisor=1.0 / cfg.logit_scale, tied=False, name="head",
                      params={"softcap": float(cfg.logit_softcap or 0.0)}),
        max_positions=0, ignorable=ignorable)
    plan.validate()
    return plan


register_architecture(NAMES, TunavikConfig, build_plan)
