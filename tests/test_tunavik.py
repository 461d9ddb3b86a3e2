"""Tunavik without a GPU: the configuration reader, the plan and its tensor list, random models on disk, the distance
buckets, layers that share one layer's pages, and hand-computed checks of the plain implementation's mechanisms."""
import json
import math
import os

import pytest
import torch

from exl3_server_b200.cache.kv import SequenceCache
from exl3_server_b200.config import ConfigError, resolve_architecture
from exl3_server_b200.config.tunavik import TunavikConfig
from exl3_server_b200.engine.model import plan_manifest
from exl3_server_b200.parts.base import KVRequest
from exl3_server_b200.parts.distance_bias import DistanceBias, bucket_starts
from exl3_server_b200.parts.normed_attention import tile_row
import plain_tunavik as P
from tunavik_configs import CONFIGS, make_tunavik


def test_config_round_trip_and_plan():
    cfg = CONFIGS["mixed"]
    obj = json.loads(json.dumps(cfg.to_dict()))
    arch = resolve_architecture(obj)
    again = arch.config_class.from_dict(obj)
    assert arch.config_class.from_dict(json.loads(json.dumps(again.to_dict()))).to_dict() == again.to_dict()
    assert again.to_dict()["layers"][0]["mixer"]["q_temp"] == {"coef": 0.5, "every": 10.0}
    plan = arch.build_plan(again)
    assert all(l.mixer.kind == "normed_attention" and l.arrangement == "outnorm" for l in plan.layers)
    assert [e.cache_from for e in plan.schedule] == [None, None, 0, 1, 0, None]
    a = plan.layers[0].mixer
    assert (a.params["qk_norm"], a.params["q_temp"], a.params["distance_bias"], a.params["sink"], a.params["bias"],
            a.params["reads_kv"], a.softmax_scale) == ("rows", (0.5, 10.0), 50, "learned", True, False, 0.21)
    assert plan.layers[3].mixer.params["reads_kv"] and plan.layers[3].mixer.params["q_temp"] is None
    ff = plan.layers[0].feed_forward
    assert ff.kind == "routed" and (ff.params["score"], ff.params["activation"], ff.params["shared_inner"]) == ("picked", "relu2", 56)
    assert plan.layers[1].feed_forward is None and plan.layers[2].feed_forward.params["shared_inner"] == 0
    assert plan.embedding.kind == "table_sinusoid" and not plan.head.tied and plan.head.params["softcap"] == 3.0
    assert math.isclose(1.0 / plan.head.input_divisor, 1.7)
    names = {s.name: s.shape for s in plan_manifest(plan)}
    assert names["embed.norm"] == (96,) and names["head"] == (211, 96) and names["l0.mix.rel"] == (-1, 4)
    assert names["l0.mix.q.norm"] == (96,) and names["l0.mix.k.norm"] == (48,) and names["l0.mix.o.b"] == (96,)
    assert names["l3.mix.q"] == (48, 96) and names["l3.mix.sink"] == (3,) and names["l3.mix.rel"] == (-1, 3)
    for gone in ("l3.mix.k", "l3.mix.v", "l3.mix.k.b", "l3.mix.v.b", "l3.mix.k.norm", "l0.mlp.correction", "l0.mlp.shared.sg",
                 "l2.mlp.shared.up", "l1.norm2"):
        assert gone not in names, gone
    assert names["l0.mlp.router.b"] == (9,) and names["l0.mlp.e8.up"] == (40, 96) and names["l0.mlp.shared.down"] == (96, 56)
    assert "l1.norm2" in plan.ignorable


def test_what_the_configuration_leaves_out_is_not_there():
    obj = CONFIGS["odd"].to_dict()
    for key in ("q_temp", "kv_from"):
        obj["layers"][0]["mixer"].pop(key, None)
    obj["layers"][0]["mlp"].pop("shared")
    obj["layers"][1].pop("mlp")
    obj.pop("logit_softcap")
    obj.pop("logit_scale")
    plan = resolve_architecture(obj).build_plan(TunavikConfig.from_dict(obj))
    assert plan.layers[0].mixer.params["q_temp"] is None and plan.layers[0].feed_forward.params["shared_inner"] == 0
    assert plan.layers[1].feed_forward is None and plan.head.params["softcap"] == 0.0 and plan.head.input_divisor == 1.0


@pytest.mark.parametrize("change, message", [
    (lambda o: o["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda o: o["layers"][0]["mixer"].pop("bias_max"), "bias_max"),
    (lambda o: o["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda o: o["layers"][0]["mixer"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda o: o["layers"][0]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda o: o["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda o: o["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda o: o["layers"][0]["mlp"]["router"].__setitem__("top", 10), "top"),
    (lambda o: o["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda o: o["layers"][2]["mixer"].__setitem__("kv_from", 2), "kv_from"),
    (lambda o: o["layers"][4]["mixer"].__setitem__("kv_from", 2), "kv_from"),
    (lambda o: o["layers"][3]["mixer"].__setitem__("kv_from", 0), "kv_heads"),
    (lambda o: o["norm"].pop("eps"), "eps"),
    (lambda o: o.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda o: o.__setitem__("layers", []), "layers"),
])
def test_config_errors_name_the_key(change, message):
    obj = CONFIGS["mixed"].to_dict()
    change(obj)
    with pytest.raises(ConfigError, match=message):
        TunavikConfig.from_dict(obj)


def test_random_model_on_disk_matches_its_manifest(tmp_path):
    folder = make_tunavik("mixed", str(tmp_path / "m"))
    w = P.read_weights(folder)
    cfg = json.load(open(os.path.join(folder, "config.json")))
    assert cfg["architecture"] == "Tunavik" and len(cfg["layers"]) == 6
    plan = resolve_architecture(cfg).build_plan(TunavikConfig.from_dict(cfg))
    for s in plan_manifest(plan):
        assert s.name in w and all(e in (-1, g) for g, e in zip(w[s.name].shape, s.shape)), s.name
    assert sorted({w[f"l{i}.mix.rel"].shape[0] for i in range(6)}) == [2, 6, 9, 16, 26, 40]
    logits = P.PlainTunavik(folder).logits([1, 2, 3, 4])
    assert logits.shape == (4, 211) and torch.isfinite(logits).all()


@pytest.mark.parametrize("rows, limit", [(16, 50), (40, 300), (9, 21), (2, 64), (26, 160), (6, 97), (8, 64), (12, 48), (10, 5.5),
                                         (7, 100.25), (16, 9), (3, 2), (64, 1000)])
def test_buckets_by_distance(rows, limit):
    """The starts of the buckets against the formula distance by distance, also where a distance is an exact power (8 rows
    up to 64: buckets of 4, 8, 16 and 32 positions) and where geometric buckets are shorter than one position."""
    starts = bucket_starts(rows, limit)
    assert len(starts) == rows and starts == sorted(starts)
    for n in range(int(limit) + 20):
        mine = max(b for b in range(rows) if starts[b] <= n)
        assert mine == P.bucket(n, rows, limit), n
    if (rows, limit) == (8, 64):
        assert starts == [0, 1, 2, 3, 4, 8, 16, 32]
    with pytest.raises(ValueError, match="largest distance"):
        bucket_starts(rows, rows // 2)


def test_biases_are_kept_relative_to_the_far_ones():
    rel = torch.randn(10, 3, dtype=torch.float64)
    b = DistanceBias(rel, 40)
    assert torch.equal(b.far, rel[-1]) and b.near.shape == (3, bucket_starts(10, 40)[-1])
    for n in range(60):
        got = b.far + (b.near[:, n] if n < b.near.shape[1] else 0.0)
        assert torch.allclose(got, rel[P.bucket(n, 10, 40)], atol=1e-12), n
    one = DistanceBias(rel[:1], 5)                     # a table of one row: the same for every key
    assert one.near.shape == (3, 0) and torch.equal(one.far, rel[0])


def test_rows_of_the_tensor_core_kernels():
    assert [tile_row(*p) for p in ((64, 64), (40, 16), (16, 65), (128, 8), (129, 8), (8, 200))] == [64, 64, 128, 128, 0, 0]


def test_readers_share_their_owners_pages():
    own, reader = KVRequest(2, 24, value_dim=16), KVRequest(2, 24, value_dim=16)
    cache = SequenceCache([(own, None, None), (KVRequest(3, 16, value_dim=40), None, None), (reader, None, 0),
                           (reader, None, 0)], max_tokens=640, device="cpu", dtype=torch.float32)
    assert len(cache.groups) == 2 and cache.groups[0].k.shape[0] == 1          # one layer of storage for three entries
    s = cache.open()
    cache.reserve({s: 130})
    cache.commit(s, 130)
    tables = [torch.tensor(t) for t in cache.block_tables([s])]
    views = [cache.view(i, tables) for i in range(4)]
    assert [v.owns for v in views] == [True, True, False, False]
    assert views[2].k.data_ptr() == views[0].k.data_ptr() and views[3].v.data_ptr() == views[0].v.data_ptr()
    cache.truncate(s, 70)
    cache.close(s)
    cache.check()
    with pytest.raises(Exception, match="head shapes"):
        SequenceCache([(own, None, None), (KVRequest(2, 32, value_dim=16), None, 0)], max_tokens=64, device="cpu")


def test_plain_sinusoids_temperature_and_buckets_by_hand():
    s = P.sinusoids(3, 5)
    assert s[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0]
    f1, f2 = 10000.0 ** (-2.0 / 5), 10000.0 ** (-4.0 / 5)
    assert torch.allclose(s[2], torch.tensor([math.sin(2.0), math.cos(2.0), math.sin(2 * f1), math.cos(2 * f1), math.sin(2 * f2)],
                                             dtype=P.F))
    t = P.temperature(7, 0.5, 3)                       # p + 1 = 1, 2 | 3, 4, 5 | 6, 7
    assert torch.allclose(t, 1.0 + 0.5 * torch.log(torch.tensor([1.0, 1, 2, 2, 2, 3, 3], dtype=P.F)))
    assert [P.bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 5000)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]


def test_plain_attention_by_hand():
    """One head of one feature, two tokens: a query and a key are their signs after the norm."""
    one, zero = torch.ones(1, 1, dtype=P.F), torch.zeros(1, dtype=P.F)
    w = {"p.q": one, "p.k": one, "p.v": one, "p.o": 2.0 * one, "p.q.b": zero, "p.k.b": zero, "p.v.b": zero + 0.25,
         "p.o.b": zero - 1.0, "p.q.norm": zero + 1.5, "p.k.norm": zero + 2.0, "p.sink": zero + 0.5,
         "p.rel": torch.tensor([[0.3], [-0.7]], dtype=P.F)}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.5, "bias_max": 4, "q_temp": {"coef": 0.1, "every": 2}}
    h = torch.tensor([[1.0], [-3.0]], dtype=P.F)
    y = P.attention(h, w, "p.", m, 0.0, P.keys_and_values(h, w, "p.", m, 0.0))
    e00 = math.exp(1.5 * 2.0 * 0.5 + 0.3)
    assert math.isclose(float(y[0]), 2.0 * (e00 * 1.25) / (e00 + math.exp(0.5)) - 1.0)
    temp = 1.0 + 0.1 * math.log(2.0)                   # p = 1: floor(2 / 2) + 1
    e10, e11 = math.exp(-1.5 * temp * 2.0 * 0.5 - 0.7), math.exp(1.5 * temp * 2.0 * 0.5 + 0.3)
    assert math.isclose(float(y[1]), 2.0 * (e10 * 1.25 + e11 * -2.75) / (e10 + e11 + math.exp(0.5)) - 1.0)
    # one norm over both heads together: the larger head keeps its size relative to the smaller
    w2 = {"p.k": torch.tensor([[3.0], [4.0]], dtype=P.F), "p.k.b": torch.zeros(2, dtype=P.F), "p.k.norm": torch.ones(2, dtype=P.F),
          "p.v": torch.zeros(2, 1, dtype=P.F), "p.v.b": torch.zeros(2, dtype=P.F)}
    k, _ = P.keys_and_values(h[:1], w2, "p.", {"kv_heads": 2, "dim": 1, "vdim": 1}, 0.0)
    assert torch.allclose(k.flatten(), torch.tensor([3.0, 4.0], dtype=P.F) / math.sqrt(12.5))


def test_plain_router_by_hand():
    picks, wts, margin = P.route(torch.tensor([0.1, 2.0, -1.0, 1.5], dtype=P.F), 2)
    assert picks == [1, 3] and math.isclose(margin, 1.4) and math.isclose(float(wts[0]), 1 / (1 + math.exp(-0.5)))
    w = {"p.router": torch.eye(2, dtype=P.F), "p.router.b": torch.tensor([0.0, 10.0], dtype=P.F)}
    for e in (0, 1):
        w.update({f"p.e{e}.up": torch.tensor([[1.0, -1.0]], dtype=P.F), f"p.e{e}.down": torch.tensor([[1.0 + e], [0.0]], dtype=P.F)})
    w.update({"p.shared.up": torch.tensor([[0.0, 1.0]], dtype=P.F), "p.shared.down": torch.tensor([[0.0], [5.0]], dtype=P.F)})
    mlp = {"expert": {"ff": 1}, "router": {"experts": 2, "top": 1}, "shared": {"ff": 1}}
    y = P.mixture_of_experts(torch.tensor([[3.0, 1.0], [1.0, 3.0]], dtype=P.F), w, "p.", mlp)
    assert y.tolist() == [[8.0, 5.0], [0.0, 45.0]]     # the bias decides for the second expert; a single pick weighs one
