"""Soporax without a GPU: the configuration reader, the plan, its schedule and tensor list, random models on disk, frequency
tables, passes with caches of their own, and hand-computed checks of the plain implementation's mechanisms."""
import json
import math
import os

import pytest
import torch

from exl3_server_b200.cache.kv import SequenceCache
from exl3_server_b200.config import ConfigError, resolve_architecture
from exl3_server_b200.config.soporax import SoporaxConfig
from exl3_server_b200.engine.model import Model, plan_manifest
from exl3_server_b200.parts.base import BuildContext
from exl3_server_b200.parts.position import RotaryPosition
from exl3_server_b200.parts.spec import PositionSpec, ScheduleEntry
from exl3_server_b200.weights.loader import load_tensors
import plain_soporax as P
from soporax_configs import CONFIGS, bands, make_soporax, ramp


def plan_of(name):
    obj = CONFIGS[name].to_dict()
    return resolve_architecture(obj).build_plan(SoporaxConfig.from_dict(obj))


def test_config_round_trip_and_plan():
    obj = json.loads(json.dumps(CONFIGS["mixed"].to_dict()))
    arch = resolve_architecture(obj)
    again = arch.config_class.from_dict(obj)
    assert arch.config_class.from_dict(json.loads(json.dumps(again.to_dict()))).to_dict() == again.to_dict()
    plan = arch.build_plan(again)
    assert all(l.arrangement == "parallel" and l.feed_forward_norm is None for l in plan.layers)
    assert [l.mixer.kind for l in plan.layers] == ["normed_attention", "latent_attention", "normed_attention",
                                                   "latent_attention", "normed_attention", "normed_attention"]
    a, w, z = plan.layers[0].mixer, plan.layers[2].mixer, plan.layers[1].mixer
    assert (a.params["bias"], a.params["sink"], a.params["gate"], a.window, a.softmax_scale) == ("qkv", True, "head", 0, 0.21)
    assert a.position.params == {"layout": "interleaved", "bands": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 40.0}}
    assert (w.params["qk_norm"], w.params["sink"], w.window, w.position) == ("unit", "learned", 37, None)
    assert z.params["gate"] == "element" and z.position.params["yarn"]["factor"] == 6.0 and z.position.dims == 16
    ff = [l.feed_forward for l in plan.layers]
    assert ff[4] is None and ff[1].kind == "clamped_glu" and ff[1].params["limit"] == 0.6
    assert ff[2].kind == "table_routed" and (ff[2].params["experts"], ff[2].params["top"], ff[2].params["expert"]) == (5, 3, "glu")
    assert plan.head.tied and plan.final_norm.params["scale"] == 1.7
    names = {s.name: s for s in plan_manifest(plan)}
    assert names["loop.step"].shape == (4, 96) and names["l2.mlp.table"].shape == (211, 3) and names["l2.mlp.table"].kind == "int"
    assert names["l0.mix.g"].shape == (6, 96) and names["l1.mix.g"].shape == (200, 96) and names["l2.mix.sink"].shape == (4,)
    assert names["l0.mlp.e8.gate"].shape == (40, 96) and names["l1.mlp.down"].shape == (96, 72)
    for gone in ("head", "l0.norm2", "l2.mlp.router", "l0.mix.o.b", "l2.mix.q.b", "l0.mix.sink", "l2.mix.g", "l4.mlp.table"):
        assert gone not in names, gone


def test_the_schedule_runs_the_loop_pass_by_pass():
    e = plan_of("mixed").schedule
    assert [x.layer for x in e] == [0, 1, 2, 1, 2, 1, 2, 1, 2, 3, 4, 5]
    assert [(x.add_embedding, x.add_vector) for x in e] == [(False, None), (False, 0), (False, None), (True, 1), (False, None),
                                                            (True, 2), (False, None), (True, 3)] + [(False, None)] * 4
    assert [x.layer for x in plan_of("odd").schedule] == [0, 1, 0, 1, 0, 1, 2, 3]
    assert [x.layer for x in plan_of("wide").schedule] == [0, 1, 2, 3, 4, 5, 5, 5]
    once = plan_of("once")
    assert once.entry_vectors is None and [x.layer for x in once.schedule] == [0, 1]
    assert "loop.step" not in {s.name for s in plan_manifest(once)}
    for name, c in CONFIGS.items():
        runs = P.layer_runs(c.to_dict())
        assert [(x.layer, x.add_vector) for x in plan_of(name).schedule] == runs, name
    broken = plan_of("mixed")
    broken.schedule[3] = ScheduleEntry(layer=1, add_vector=4)
    with pytest.raises(ValueError, match="adds vector 4"):
        broken.validate()


def test_every_pass_has_keys_and_values_of_its_own(tmp_path):
    folder = make_soporax("mixed", str(tmp_path / "m"))
    plan = plan_of("mixed")
    model = Model(plan, load_tensors(folder, plan_manifest(plan), torch.float32), torch.float32, "cpu")
    cache = SequenceCache(model.cache_requests(), max_tokens=640, device="cpu", dtype=torch.float32)
    s = cache.open()
    cache.reserve({s: 130})
    cache.commit(s, 130)
    tables = [torch.tensor(t) for t in cache.block_tables([s])]
    views = [cache.view(i, tables) for i in range(len(plan.schedule))]
    assert all(v.owns for v in views) and len({v.k.data_ptr() for v in views}) == len(views)
    # the window's group gives back the page that no later query can see, whichever pass it belongs to
    assert sum(int(t[0, 0]) < 0 for t in tables) >= 1
    cache.close(s)
    cache.check()
    assert [p[2] for p in model.blocks[0].feed_forward.peers] == [2, 3, 1]      # all table layers of the model know each other


def test_what_the_configuration_leaves_out_is_not_there():
    obj = CONFIGS["mixed"].to_dict()
    obj["layers"][2]["mixer"].pop("mask")
    obj["layers"][0]["mixer"]["rot"].pop("scaling")
    obj["layers"][5]["mixer"].pop("rot")
    obj["layers"][1].pop("mlp")
    obj.pop("loop")
    obj.pop("logit_scale")
    plan = resolve_architecture(obj).build_plan(SoporaxConfig.from_dict(obj))
    assert plan.layers[2].mixer.window == 0 and plan.layers[0].mixer.position.params == {"layout": "interleaved"}
    assert plan.layers[5].mixer.position is None and plan.layers[1].feed_forward is None
    assert plan.entry_vectors is None and plan.final_norm.params["scale"] == 1.0 and len(plan.schedule) == 6


@pytest.mark.parametrize("change, message", [
    (lambda o: o["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda o: o["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda o: o["layers"][0]["mixer"]["rot"].__setitem__("dims", 26), "dims"),
    (lambda o: o["layers"][0]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda o: o["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda o: o["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda o: o["layers"][2]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda o: o["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda o: o["layers"][0]["mlp"].__setitem__("kind", "wide"), "kind"),
    (lambda o: o["layers"][0]["mlp"]["router"].__setitem__("top", 10), "top"),
    (lambda o: o["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda o: o["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda o: o["loop"].__setitem__("stop", 7), "loop"),
    (lambda o: o["loop"].__setitem__("stop", 1), "loop"),
    (lambda o: o["loop"].pop("times"), "times"),
    (lambda o: o["norm"].pop("eps"), "eps"),
    (lambda o: o.__setitem__("layers", []), "layers"),
])
def test_config_errors_name_the_key(change, message):
    obj = CONFIGS["mixed"].to_dict()
    change(obj)
    with pytest.raises(ConfigError, match=message):
        SoporaxConfig.from_dict(obj)


def test_random_model_on_disk_matches_its_manifest(tmp_path):
    folder = make_soporax("mixed", str(tmp_path / "m"))
    w = P.read_weights(folder)
    cfg = json.load(open(os.path.join(folder, "config.json")))
    assert cfg["architecture"] == "Soporax" and len(cfg["layers"]) == 6
    plan = resolve_architecture(cfg).build_plan(SoporaxConfig.from_dict(cfg))
    for s in plan_manifest(plan):
        assert s.name in w and tuple(w[s.name].shape) == s.shape, s.name
    table = w["l2.mlp.table"]
    assert int(table.min()) == 0 and int(table.max()) == 4 and all(len(set(row)) == 3 for row in table.tolist())
    logits = P.PlainSoporax(folder).logits([1, 2, 3, 4])
    assert logits.shape == (4, 211) and torch.isfinite(logits).all()


def test_a_table_that_names_no_expert_is_refused(tmp_path):
    folder = make_soporax("only_moe", str(tmp_path / "m"))
    plan = plan_of("only_moe")
    tensors = load_tensors(folder, plan_manifest(plan), torch.float32)
    tensors["l0.mlp.table"][5, 1] = 14
    with pytest.raises(ValueError, match="14 experts"):
        Model(plan, tensors, torch.float32, "cpu")


@pytest.mark.parametrize("dims, base, s", [(64, 10000.0, bands(8.0, 1.0, 4.0, 1000)), (16, 500.0, bands(4.0, 2.0, 3.0, 40)),
                                           (2, 10.0, bands(2.0, 1.0, 4.0, 20)), (128, 500000.0, bands(32.0, 1.0, 4.0, 8192))])
def test_frequencies_scaled_by_bands(dims, base, s):
    got = RotaryPosition.frequencies(PositionSpec(kind="rope", dims=dims, theta=base, params={"bands": s}))
    want = torch.tensor(P.banded_frequencies(dims, base, s), dtype=torch.float64)
    assert torch.allclose(got, want, rtol=1e-13, atol=0.0)
    ratio = torch.tensor(P.base_frequencies(dims, base), dtype=torch.float64) / got
    assert float(ratio.min()) >= 1.0 - 1e-12 and float(ratio.max()) <= s["factor"] + 1e-9


def test_the_two_scalings_exclude_each_other():
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"))
    for one, m in (({"bands": bands(2.0, 1.0, 4.0, 64)}, 1.0), ({"yarn": ramp(2.0, 64, 8.0, 1.0)}, 0.1 * math.log(2.0) + 1.0)):
        assert math.isclose(RotaryPosition(PositionSpec(kind="rope", dims=8, params=one), 8, ctx).mscale, m)
    with pytest.raises(ValueError, match="two ways"):
        RotaryPosition(PositionSpec(kind="rope", dims=8, params={"bands": bands(2.0, 1.0, 4.0, 64), "yarn": ramp(2.0, 64, 8.0, 1.0)}), 8, ctx)


def test_plain_frequencies_by_hand():
    # wavelengths 2 pi and 20 pi; a context of 40 positions with bounds at 40 / 4 = 10 and 40 / 1 = 40
    f = P.banded_frequencies(4, 100.0, bands(4.0, 1.0, 4.0, 40))
    assert f[0] == 1.0 and math.isclose(f[1], 0.1 / 4.0)
    f = P.banded_frequencies(4, 100.0, bands(4.0, 0.5, 1.0, 40))       # 20 pi = 62.8 lies between 40 and 80
    part = (40 / (20 * math.pi) - 0.5) / 0.5
    assert math.isclose(f[1], (1 - part) * 0.1 / 4.0 + part * 0.1)
    f, m = P.ramped_frequencies(4, 100.0, ramp(3.0, 40, 2.0, 0.01))
    lo, hi = 0, min(math.ceil(4 * math.log(40 / (2 * math.pi * 0.01)) / (2 * math.log(100.0))), 3)
    assert hi == 3 and f[0] == 1.0 and math.isclose(f[1], 0.1 / 3 * (1 / 3) + 0.1 * (2 / 3)) and math.isclose(m, 0.1 * math.log(3.0) + 1)
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0, 7.0]] * 3, dtype=P.F)
    y = P.rotate_neighbours(x, [0.5, 0.25], 2.0)
    assert torch.allclose(y[2], torch.tensor([2 * math.cos(1.0), 2 * math.sin(1.0), -4 * math.sin(0.5), 4 * math.cos(0.5), 7.0], dtype=P.F))


def test_plain_attention_by_hand():
    """One head of one feature, two tokens: a query and a key are their signs after the norm."""
    one = torch.ones(1, 1, dtype=P.F)
    w = {"p.q": one, "p.k": one, "p.v": one, "p.o": 2.0 * one, "p.sink": torch.tensor([0.5], dtype=P.F)}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.5, "mask": {"size": 2}}
    h = torch.tensor([[1.0], [-3.0], [2.0]], dtype=P.F)
    y = P.windowed_attention(h, w, "p.", m, 0.0)
    assert math.isclose(float(y[0]), 2.0 * math.exp(0.5) / (2.0 * math.exp(0.5)))
    same, other = math.exp(0.5), math.exp(-0.5)
    assert math.isclose(float(y[1]), 2.0 * (other * 1.0 + same * -3.0) / (same + other + math.exp(0.5)))
    assert math.isclose(float(y[2]), 2.0 * (other * -3.0 + same * 2.0) / (same + other + math.exp(0.5)))   # the first is out of sight
    zero = torch.zeros(1, dtype=P.F)
    w = {"p.q": one, "p.k": one, "p.v": one, "p.o": one, "p.q.b": zero + 1.0, "p.k.b": zero, "p.v.b": zero - 1.0, "p.g": 0.5 * one}
    y = P.rotated_attention(h[:2], w, "p.", {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.25}, 0.0)
    s = [math.exp(-2.0 * 1.0 * 0.25), math.exp(-2.0 * -3.0 * 0.25)]
    assert math.isclose(float(y[1]), (s[0] * 0.0 + s[1] * -4.0) / (1.0 + s[0] + s[1]) / (1.0 + math.exp(1.5)))


def test_plain_latent_attention_by_hand():
    one = torch.ones(1, 1, dtype=P.F)
    w = {"p.dq": 3.0 * one, "p.dq.norm": torch.tensor([2.0], dtype=P.F), "p.uq": 0.5 * one,
         "p.dkv": one, "p.dkv.norm": torch.tensor([1.5], dtype=P.F), "p.uk": 2.0 * one, "p.uv": 4.0 * one, "p.g": one, "p.o": one}
    m = {"heads": 1, "dim": 1, "rot_dim": 0, "vdim": 1, "q_rank": 1, "kv_rank": 1, "scale": 0.1}
    y = P.latent_attention(torch.tensor([[1.0], [-3.0]], dtype=P.F), w, "p.", m, 0.0)
    # latents are signs times their weights: c = 1.5, -1.5; q = 1, -1; k = 3, -3; v = 6, -6
    a, b = math.exp(-0.3), math.exp(0.3)
    assert math.isclose(float(y[1]), (a * 6.0 - b * 6.0) / (a + b) / (1.0 + math.exp(3.0)))


def test_plain_feed_forwards_and_loop_by_hand():
    w = {"p.gate": torch.tensor([[1.0]], dtype=P.F), "p.up": torch.tensor([[-2.0]], dtype=P.F), "p.down": torch.tensor([[3.0]], dtype=P.F)}
    y = P.clamped_feed_forward(torch.tensor([[5.0], [-5.0]], dtype=P.F), w, "p.", 0.75)
    assert math.isclose(float(y[0]), 3.0 * 0.75 / (1 + math.exp(-1.702 * 0.75)) * 0.25)
    assert math.isclose(float(y[1]), 3.0 * -5.0 / (1 + math.exp(1.702 * 5.0)) * 1.75)        # the gate has no lower bound
    w = {"p.table": torch.tensor([[1, 0], [2, 1]])}
    for e in range(3):
        w.update({f"p.e{e}.gate": torch.tensor([[1.0]], dtype=P.F), f"p.e{e}.up": torch.tensor([[1.0 + e]], dtype=P.F),
                  f"p.e{e}.down": torch.tensor([[1.0]], dtype=P.F)})
    y = P.experts_by_table(torch.tensor([[2.0], [2.0]], dtype=P.F), w, "p.", [1, 0])
    silu = 2.0 / (1 + math.exp(-2.0))
    assert torch.allclose(y.flatten(), torch.tensor([silu * 2.0 * 2.5, silu * 2.0 * 1.5], dtype=P.F))
    # a model whose layer adds nothing: only the passes' vectors and the embedding remain
    zero = torch.zeros(2, 2, dtype=P.F)
    w = {"embed": torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=P.F), "loop.step": torch.tensor([[10.0, 0.0], [0.0, 20.0]], dtype=P.F),
         "l0.norm1": torch.ones(2, dtype=P.F), "final.norm": torch.ones(2, dtype=P.F), "l0.mix.sink": torch.zeros(1, dtype=P.F),
         **{f"l0.mix.{n}": zero for n in "qkvo"}}
    cfg = {"norm": {"eps": 1e-9}, "loop": {"start": 0, "stop": 1, "times": 2}, "logit_scale": 3.0,
           "layers": [{"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0}, "mlp": None}]}
    seen = []
    out = P.forward(cfg, w, [1], seen)
    assert seen[0].tolist() == [[13.0, 4.0]] and seen[1].tolist() == [[16.0, 28.0]]
    x = torch.tensor([16.0, 28.0], dtype=P.F)
    assert torch.allclose(out[0], 3.0 * w["embed"] @ (x / torch.sqrt((x * x).mean())))
