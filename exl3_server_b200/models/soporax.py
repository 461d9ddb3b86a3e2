"""The Soporax decoder as a plan of parts.

Every layer runs its mixer and its feed-forward side by side on the output of one RMS norm (``parallel`` arrangement).
Layers come from the configuration's list:

* ``attention``: grouped-query attention over a window without positions, unit-length queries and keys, a learned sink per
  head (``normed_attention``);
* ``attention_2``: causal grouped-query attention with biases on q, k and v, rotary positions on neighbouring features with
  frequencies scaled by bands of wavelengths, one added to the softmax's denominator and a gate per head
  (``normed_attention``);
* ``latent_attention``: queries, keys and values through latents, one cached row per token, rotary positions on neighbouring
  features with a stretched frequency table (YaRN), a gate per output feature (``latent_attention``).

Feed-forwards: ``dense`` has a bounded gate (``clamped_glu``); ``moe`` has gated experts that a table picks by the token's id
(``table_routed``); or none.

A group of layers may run several times (``loop``): the schedule lists it once a pass, every pass with keys and values of its
own.  A pass begins by adding a learned vector of its own to the residual and, from the second pass on, the embedding's
output.  The head is the embedding table; the logits are multiplied by a constant, which rides on the last norm's weight.

Tensor names: ``embed``, ``loop.step``, ``final.norm`` and, per layer ``l<i>``: ``norm1``, ``mix.*`` and ``mlp.*`` (see the
parts' modules).
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.soporax import SoporaxConfig
from ..parts.spec import (EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerSpec, MixerSpec, ModelPlan, NormSpec, PositionSpec,
                          ScheduleEntry)

NAMES = ("Soporax", "soporax")


def _norm(cfg: SoporaxConfig, scale: float = 1.0) -> NormSpec:
    return NormSpec(kind="rms", width=cfg.width, eps=cfg.norm_eps, params={"suffix": "", "scale": scale})


def _position(m: dict, scaling: str):
    rot = m.get("rot")
    if not rot or rot["dims"] == 0:
        return None
    params = {"layout": "interleaved"}
    if rot.get("scaling"):
        params[scaling] = dict(rot["scaling"])
    return PositionSpec(kind="rope", dims=rot["dims"], theta=rot["base"], params=params)


def _mixer(cfg: SoporaxConfig, kind: str, m: dict) -> MixerSpec:
    if kind == "latent_attention":
        return MixerSpec(kind="latent_attention", width=cfg.width, heads=m["heads"], softmax_scale=m["scale"],
                         position=_position(m, "yarn"),
                         params={"norm_eps": cfg.norm_eps, "gate": "element",
                                 **{k: m[k] for k in ("dim", "rot_dim", "vdim", "q_rank", "kv_rank")}})
    params = {"value_dim": m["vdim"], "norm_eps": cfg.norm_eps, "tile_rows": True}
    window = 0
    if kind == "attention":
        params.update(qk_norm="unit", sink="learned")
        window = m["mask"]["size"] if m.get("mask") else 0
    else:
        params.update(bias="qkv", sink=True, gate="head")
    return MixerSpec(kind="normed_attention", width=cfg.width, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"],
                     window=window, softmax_scale=m["scale"], position=_position(m, "bands"), params=params)


def _feed_forward(cfg: SoporaxConfig, mlp: dict) -> FeedForwardSpec:
    if mlp["kind"] == "dense":
        return FeedForwardSpec(kind="clamped_glu", width=cfg.width, inner=mlp["ff"], params={"limit": mlp["limit"]})
    return FeedForwardSpec(kind="table_routed", width=cfg.width, inner=mlp["expert"]["ff"],
                           params={"vocab": cfg.vocab, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
                                   "expert": "glu", "activation": "silu"})


def _schedule(cfg: SoporaxConfig):
    """The layers in the order they run; a pass over the loop's layers begins with what joins the residual."""
    n = len(cfg.layers)
    if cfg.loop is None:
        return [ScheduleEntry(layer=i) for i in range(n)]
    start, stop, times = (cfg.loop[k] for k in ("start", "stop", "times"))
    out = [ScheduleEntry(layer=i) for i in range(start)]
    for t in range(times):
        out.append(ScheduleEntry(layer=start, add_embedding=t > 0, add_vector=t))
        out += [ScheduleEntry(layer=i) for i in range(start + 1, stop)]
    return out + [ScheduleEntry(layer=i) for i in range(stop, n)]


def build_plan(cfg: SoporaxConfig) -> ModelPlan:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        layers.append(LayerSpec(
            arrangement="parallel", mixer=_mixer(cfg, layer.type, layer.mixer),
            feed_forward=_feed_forward(cfg, layer.mlp) if layer.mlp is not None else None, mixer_norm=_norm(cfg),
            feed_forward_norm=None, residual_scale=1.0,
            names={"mixer": p + "mix.", "feed_forward": p + "mlp.", "mixer_norm": p + "norm1"}))
    plan = ModelPlan(
        architecture=cfg.architecture,
        embedding=EmbeddingSpec(vocab=cfg.vocab, width=cfg.width, scale=1.0, name="embed"), layers=layers,
        schedule=_schedule(cfg), final_norm=_norm(cfg, float(cfg.logit_scale)), final_norm_name="final.norm",
        head=HeadSpec(vocab=cfg.vocab, width=cfg.width, input_divisor=1.0, tied=True, name="embed"),
        max_positions=0, entry_vectors=("loop.step", cfg.loop["times"]) if cfg.loop is not None else None)
    plan.validate()
    return plan


register_architecture(NAMES, SoporaxConfig, build_plan)
