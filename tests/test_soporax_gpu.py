"""The Soporax decoder in the engine against the plain implementation (tests/plain_soporax.py): each mechanism alone, whole
prompts against token-by-token decoding, portions, unequal batches with slots and pages used again, keys far back, at page
borders and at a window's edge, first tokens, long decoding, passes of a loop, generation through the entry point, the
replay program; float32 and bfloat16, on configurations that differ in every size and option.  Experts are picked by token
ids, so no rounding changes a choice: every position is held to the bound in both types."""
import json
import os
import shutil
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import TOL, batched_trace, random_requests, rel_err, run_trace, tail_trace, whole_trace
import plain_soporax as P
from plain_soporax import PlainSoporax
from soporax_configs import CONFIGS, make_soporax

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
LENGTHS = {"mixed": [1, 2, 9, 64, 65, 150], "odd": [1, 3, 20, 64, 66, 131], "wide": [3, 17, 63, 128, 129, 300]}
ONLY_LENGTHS = [1, 2, 31, 64, 129, 140]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("soporax")
    return {name: make_soporax(name, str(root / name)) for name in CONFIGS}


_plain = {}


def plain(folder):
    if folder not in _plain:
        _plain[folder] = PlainSoporax(folder)
    return _plain[folder]


def engine_for(folder, dtype, max_tokens=2048):
    from exl3_server_b200 import Engine
    return Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens)


def requests_for(name, lengths, seed):
    return random_requests(CONFIGS[name].vocab, lengths, seed=seed)


def close_enough(got, want, dtype, what):
    assert got.shape == want.shape, what
    assert np.isfinite(got).all(), what
    err = np.max(np.abs(got.astype(np.float64) - want.astype(np.float64)), axis=1) / max(1e-30, np.max(np.abs(want)))
    bad = err > TOL[dtype]
    assert not bad.any(), (f"{what}: differs from the plain implementation by {err.max():.3e} (bound {TOL[dtype]:.0e}); "
                           f"first wrong position {int(np.argmax(bad))} of {len(err)}")


def check(got, want, dtype, what):
    assert set(got) == set(want)
    for rid in want:
        close_enough(got[rid], want[rid], dtype, f"{what}, request {rid}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in CONFIGS if not n.startswith("random")])
def test_whole_decoded_and_batched(folders, name, dtype):
    folder = folders[name]
    requests = requests_for(name, LENGTHS.get(name, ONLY_LENGTHS), seed=3)
    pm = plain(folder)
    want = {rid: pm.logits(t).numpy() for rid, t in requests.items()}
    eng = engine_for(folder, dtype)
    check(run_trace(eng, whole_trace(requests)), want, dtype, "whole")
    check(run_trace(eng, tail_trace(requests, 45)), want, dtype, "last 45 one by one")
    # everything but the first token decoded: the prompt path and the one-token path must walk the same sums
    short = {rid: t for rid, t in requests.items() if len(t) <= 70}
    check(run_trace(eng, tail_trace(short, 1000)), {rid: want[rid] for rid in short}, dtype, "token by token")
    ids = list(requests)
    # two batches one after the other, so that slots and pages are used again
    batches = [[ids[5], ids[0], ids[2], ids[3]], [ids[1], ids[4], ids[0]]]
    prompt_len = {rid: max(1, len(requests[rid]) - k) for rid, k in zip(ids, (0, 1, 4, 40, 33, 70))}
    check(run_trace(eng, batched_trace(requests, batches, prompt_len)),
          {rid: want[rid] for b in batches for rid in b}, dtype, "batched")
    assert eng.cache.tokens_held() == 0
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in CONFIGS if n.startswith("random")])
def test_configurations_drawn_from_a_seed(folders, name, dtype):
    """Layer orders, sizes, counts and constants that nobody chose: whole prompts, the last tokens one by one, and
    a batch of unequal requests decoded together."""
    folder = folders[name]
    requests = requests_for(name, [1, 2, 40, 66, 150], seed=41)
    pm = plain(folder)
    want = {rid: pm.logits(t).numpy() for rid, t in requests.items()}
    eng = engine_for(folder, dtype)
    check(run_trace(eng, whole_trace(requests)), want, dtype, "whole")
    check(run_trace(eng, tail_trace(requests, 70)), want, dtype, "last 70 one by one")
    ids = list(requests)
    prompt_len = {rid: max(1, len(requests[rid]) - k) for rid, k in zip(ids, (0, 1, 35, 3, 80))}
    check(run_trace(eng, batched_trace(requests, [ids[::-1]], prompt_len)), want, dtype, "batched")
    assert eng.cache.tokens_held() == 0
    eng.check_kernels()


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_float32_cuttings_agree_closely(folders, name):
    requests = requests_for(name, LENGTHS[name], seed=5)
    eng = engine_for(folders[name], "float32")
    a = run_trace(eng, whole_trace(requests))
    b = run_trace(eng, tail_trace(requests, 32))
    for rid in requests:
        assert rel_err(b[rid], a[rid]) <= 2e-6, rid


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_portions_of_a_prompt(folders, name, dtype):
    """A prompt fed in portions of many sizes, down to one and two tokens, some ending on a page border, one long enough for
    the experts to take the many-rows product."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    toks = requests_for(name, [430], seed=9)["r0"]
    want = plain(folder).logits(toks).numpy()
    eng = engine_for(folder, dtype)
    for cuts in ([2, 2, 60, 3, 61, 2, 100, 200], [64, 64, 2, 37, 63, 200], [7, 121, 2, 2, 2, 96, 199, 1], [429, 1],
                 [50, 50, 50, 130, 150], [1, 300, 129], [1, 1, 1, 2, 1, 3, 421]):
        assert sum(cuts) == len(toks)
        s = eng.open()
        got, at = [], 0
        for n in cuts:
            got.append(eng.step([StepEntry(s, toks[at:at + n], "all")]).float().cpu().numpy())
            at += n
        eng.close(s)
        close_enough(np.concatenate(got), want, dtype, f"portions {cuts}")
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_portions_in_one_batch(folders, dtype):
    """Rows that go on by portions of different sizes in the same steps, beside a row that starts."""
    from exl3_server_b200 import StepEntry
    folder = folders["mixed"]
    reqs = requests_for("mixed", [150, 90, 40], seed=13)
    pm = plain(folder)
    want = {r: pm.logits(t).numpy() for r, t in reqs.items()}
    eng = engine_for(folder, dtype)
    sa, sb = eng.open(), eng.open()
    got = {r: [] for r in reqs}
    out = eng.step([StepEntry(sa, reqs["r0"][:70], "all"), StepEntry(sb, reqs["r1"][:3], "all")]).float().cpu().numpy()
    got["r0"].append(out[:70]); got["r1"].append(out[70:])
    sc = eng.open()
    out = eng.step([StepEntry(sb, reqs["r1"][3:66], "all"), StepEntry(sc, reqs["r2"], "all"),
                    StepEntry(sa, reqs["r0"][70:72], "all")]).float().cpu().numpy()
    got["r1"].append(out[:63]); got["r2"].append(out[63:103]); got["r0"].append(out[103:])
    eng.close(sc)
    out = eng.step([StepEntry(sa, reqs["r0"][72:], "all"), StepEntry(sb, reqs["r1"][66:], "all")]).float().cpu().numpy()
    got["r0"].append(out[:78]); got["r1"].append(out[78:])
    for r in reqs:
        close_enough(np.concatenate(got[r]), want[r], dtype, r)


def _rewrite(src, folder, change):
    os.makedirs(folder)
    shutil.copy(os.path.join(src, "config.json"), folder)
    from safetensors import safe_open
    from exl3_server_b200.weights.safetensors_io import write_safetensors
    with safe_open(os.path.join(src, "model.safetensors"), framework="pt") as f:
        tensors = {k: f.get_tensor(k) for k in f.keys()}
    tensors = {k: v.float() if v.is_floating_point() else v for k, v in tensors.items()}
    change(tensors)
    write_safetensors(os.path.join(folder, "model.safetensors"),
                      ((k, v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in tensors.items()),
                      metadata={"format": "pt"})


MARKED = 77


def _marked(src, folder):
    """A copy of a model of one layer in which one token's key stands out for every query: the last feature of the model is the
    same for every token and the one before it is on for the marked token only; queries follow the last feature, keys and values
    the one before it, in features that no position turns."""
    cfg = json.load(open(os.path.join(src, "config.json")))
    layer = cfg["layers"][0]
    m = layer["mixer"]

    def change(t):
        t["embed"][:, -2:] = 0.0
        t["embed"][:, -1] = 0.12
        t["embed"][MARKED, -2] = 0.3
        t["l0.norm1"][-2:] = 1.0
        x = lambda n: t["l0.mix." + n]
        if layer["type"] == "latent_attention":
            for name, col in (("dq", -1), ("dkv", -2)):
                x(name)[0, :] = 0.0
                x(name)[0, col] = 1.0
            x("uq").view(m["heads"], m["dim"] + m["rot_dim"], -1)[:, :m["dim"], 0] = 0.5
            x("uk")[:, 0] = 0.5
            x("uv")[:, 0] = 1.0
        else:
            turned = m["rot"]["dims"] if m.get("rot") else 0
            x("q").view(m["heads"], m["dim"], -1)[:, turned:, -1] = 1.0
            x("k").view(m["kv_heads"], m["dim"], -1)[:, turned:, -2] = 1.0
            x("v")[:, -2] = 1.0
    _rewrite(src, folder, change)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_rotated", "only_rotated_tiles", "only_latent"])
def test_a_key_that_stands_out(folders, tmp_path, name, dtype):
    """The marked key sits first, second, on both sides of page borders, hundreds of tokens back and among the last; losing it
    or reading a neighbour instead changes the logits by far more than the bound.  Whole prompts, and the last 95 tokens
    decoded one by one."""
    folder = str(tmp_path / "m")
    _marked(folders[name], folder)
    pm = PlainSoporax(folder)
    base = [t if t != MARKED else 5 for t in random_requests(CONFIGS[name].vocab, [700], seed=21)["r0"]]
    plainly = pm.logits(base).numpy()
    eng = engine_for(folder, dtype)
    for place in [0, 1, 63, 64, 127, 128, 300, 639, 640, 698]:
        toks = list(base)
        toks[place] = MARKED
        want = pm.logits(toks).numpy()
        assert rel_err(plainly[-1:], want[-1:]) > 0.15, place            # the last query sees the key
        close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, ("whole", place))
        close_enough(run_trace(eng, tail_trace({"a": toks}, 95))["a"], want, dtype, ("decoded", place))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, places, n, tail", [("only_window", [0, 13, 14, 30, 63, 64, 190, 240], 330, 120),
                                                   ("only_window_tiles", [0, 30, 55, 56, 64, 127, 180, 300], 560, 340)])
def test_a_key_at_the_windows_edge(folders, tmp_path, name, places, n, tail, dtype):
    """A key that stands out is seen by exactly as many queries as the window is long: the last that sees it and the first that
    does not differ by far more than the bound, in prompts and in decoding, wherever in a page the key lies."""
    folder = str(tmp_path / "m")
    _marked(folders[name], folder)
    size = CONFIGS[name].layers[0].mixer["mask"]["size"]
    pm, off = PlainSoporax(folder), PlainSoporax(folder)
    base = [t if t != MARKED else 5 for t in random_requests(CONFIGS[name].vocab, [n], seed=25)["r0"]]
    plainly = pm.logits(base).numpy()
    eng = engine_for(folder, dtype)
    for place in places:
        toks = list(base)
        toks[place] = MARKED
        want = pm.logits(toks).numpy()
        last = place + size - 1
        assert rel_err(plainly[last:last + 1], want[last:last + 1]) > 0.15, place
        assert rel_err(plainly[last + 1:], want[last + 1:]) < 1e-9, place
        close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, ("whole", place))
        close_enough(run_trace(eng, tail_trace({"a": toks}, tail))["a"], want, dtype, ("decoded", place))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_window", "only_window_tiles"])
def test_the_sink_counts(folders, tmp_path, name, dtype):
    """Sinks far above the scores: leaving the sink out, scaling it or giving it a value would change every row."""
    folder = str(tmp_path / "m")

    def change(t):
        t["l0.mix.sink"][:] = torch.tensor([6.0, 5.0, 7.0, 4.0])
        t["l0.mix.v"] *= 60.0
    _rewrite(folders[name], folder, change)
    pm = PlainSoporax(folder)
    toks = random_requests(128, [300], seed=33)["r0"]
    want = pm.logits(toks).numpy()
    none = dict(pm.w, **{"l0.mix.sink": torch.full((4,), -1e4, dtype=torch.float64)})
    assert rel_err(P.forward(pm.cfg, none, toks).numpy(), want) > 0.3
    eng = engine_for(folder, dtype)
    close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, "whole")
    close_enough(run_trace(eng, tail_trace({"a": toks}, 90))["a"], want, dtype, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_rotated", "only_rotated_tiles"])
def test_one_in_the_denominator_counts(folders, tmp_path, name, dtype):
    """Scores far below zero: almost all weight lies on the added one."""
    folder = str(tmp_path / "m")

    def change(t):
        t["l0.mix.q.b"][:] = 1.0
        t["l0.mix.k.b"][:] = -0.5
        t["l0.mix.v"] *= 100.0
    _rewrite(folders[name], folder, change)
    pm = PlainSoporax(folder)
    toks = random_requests(128, [200], seed=39)["r0"]
    want = pm.logits(toks).numpy()
    eng = engine_for(folder, dtype)
    close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, "whole")
    close_enough(run_trace(eng, tail_trace({"a": toks}, 90))["a"], want, dtype, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_rotated", "only_rotated_tiles", "only_latent"])
def test_gates_close_and_open(folders, tmp_path, name, dtype):
    """Gates of every size, up to shut and wide open; a gate read from the wrong column, head or feature would show."""
    folder = str(tmp_path / "m")

    def change(t):
        t["l0.mix.g"] *= 20.0
        t["l0.mix." + ("uv" if name == "only_latent" else "v")] *= 20.0
    _rewrite(folders[name], folder, change)
    pm = PlainSoporax(folder)
    toks = random_requests(128, [170], seed=51)["r0"]
    want = pm.logits(toks).numpy()
    eng = engine_for(folder, dtype)
    close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, "whole")
    close_enough(run_trace(eng, tail_trace({"a": toks}, 60))["a"], want, dtype, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_every_number_of_passes(folders, tmp_path, name, dtype):
    """One to six passes over the loop's layers; each pass's vector and the embedding's second and later additions count."""
    toks = requests_for(name, [90], seed=45)["r0"]
    for times in (1, 2, 6):
        folder = str(tmp_path / f"t{times}")

        def change(t):
            g = torch.Generator().manual_seed(times)
            t["loop.step"] = (torch.rand(times, t["loop.step"].shape[1], generator=g) - 0.5) * 0.3
        _rewrite(folders[name], folder, change)
        path = os.path.join(folder, "config.json")
        cfg = json.load(open(path))
        cfg["loop"]["times"] = times
        json.dump(cfg, open(path, "w"))
        pm = PlainSoporax(folder)
        want = pm.logits(toks).numpy()
        for lost in (dict(pm.w, **{"loop.step": torch.zeros_like(pm.w["loop.step"])}),
                     dict(pm.w, **{"loop.step": pm.w["loop.step"].roll(1, 0)})):
            assert rel_err(P.forward(pm.cfg, lost, toks).numpy(), want) > 0.02 or (times == 1 and lost["loop.step"].abs().max() > 0)
        eng = engine_for(folder, dtype)
        close_enough(run_trace(eng, whole_trace({"a": toks}))["a"], want, dtype, ("whole", times))
        close_enough(run_trace(eng, tail_trace({"a": toks}, 40))["a"], want, dtype, ("decoded", times))


def test_what_joins_the_residual_ahead_of_a_layer_of_another_arrangement():
    """Schedule entries with a vector and the embedding's output before pre-norm layers, which know nothing of them, after an
    embedding that is no row of a table, with the table's experts as one of two sublayers."""
    from exl3_server_b200 import Engine, StepEntry
    from exl3_server_b200.engine.model import Model, plan_manifest
    from exl3_server_b200.parts.spec import EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerSpec, MixerSpec, ModelPlan, NormSpec, ScheduleEntry
    from exl3_server_b200.weights.random_init import random_tensors
    W, V = 48, 60
    norm = NormSpec(kind="rms", width=W, eps=1e-5, params={"suffix": ""})
    m = {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 8, "scale": 0.4, "mask": {"size": 11}}
    mixer = MixerSpec(kind="normed_attention", width=W, heads=2, kv_heads=1, head_dim=16, window=11, softmax_scale=0.4,
                      params={"value_dim": 8, "qk_norm": "unit", "sink": "learned", "norm_eps": 1e-5})
    ff = FeedForwardSpec(kind="table_routed", width=W, inner=24, params={"vocab": V, "experts": 5, "top": 2, "expert": "glu", "activation": "silu"})
    layer = lambda i: LayerSpec(arrangement="prenorm", mixer=mixer, feed_forward=ff, mixer_norm=norm, feed_forward_norm=norm, residual_scale=0.8,
                                names={"mixer": f"l{i}.mix.", "feed_forward": f"l{i}.mlp.", "mixer_norm": f"l{i}.norm1", "feed_forward_norm": f"l{i}.norm2"})
    runs = [(0, True, 0), (1, False, None), (0, True, 1), (1, False, 2)]
    plan = ModelPlan(architecture="test", embedding=EmbeddingSpec(vocab=V, width=W, scale=2.0, name="embed", kind="table_sinusoid",
                                                                  params={"base": 10000.0}),
                     layers=[layer(0), layer(1)], schedule=[ScheduleEntry(layer=i, add_embedding=a, add_vector=v) for i, a, v in runs],
                     final_norm=norm, final_norm_name="final.norm", head=HeadSpec(vocab=V, width=W, input_divisor=1.0, tied=False, name="head"),
                     max_positions=0, entry_vectors=("steps", 3))
    tensors = dict(random_tensors(plan_manifest(plan), seed=3, std=0.15, norm_std=0.2, dtype=torch.float32))
    w = {k: (t.double() if t.is_floating_point() else t.long()) for k, t in tensors.items()}
    toks = random_requests(V, [40], seed=7)["r0"]
    at = torch.arange(40, dtype=torch.float64)[:, None] * torch.tensor([10000.0 ** (-2.0 * (i // 2) / W) for i in range(W)], dtype=torch.float64)
    start = 2.0 * w["embed"][torch.tensor(toks)] + torch.where(torch.arange(W) % 2 == 0, at.sin(), at.cos())
    x = start
    for i, add, v in runs:
        x = x + (start if add else 0) + (w["steps"][v] if v is not None else 0)
        x = x + 0.8 * P.windowed_attention(P.rms_norm(x, w[f"l{i}.norm1"], 1e-5), w, f"l{i}.mix.", m, 1e-5)
        x = x + 0.8 * P.experts_by_table(P.rms_norm(x, w[f"l{i}.norm2"], 1e-5), w, f"l{i}.mlp.", toks)
    want = (P.rms_norm(x, w["final.norm"], 1e-5) @ w["head"].T).numpy()
    for dtype in DTYPES:
        dt = getattr(torch, dtype)
        model = Model(plan, {k: (t.to("cuda:0", dt) if t.is_floating_point() else t.to("cuda:0")) for k, t in tensors.items()}, dt, "cuda:0")
        eng = Engine(model, max_tokens=512)
        s = eng.open()
        got = [eng.step([StepEntry(s, toks[:30], "all")]).float().cpu().numpy()]
        got += [eng.step([StepEntry(s, [t], "all")]).float().cpu().numpy() for t in toks[30:]]
        close_enough(np.concatenate(got), want, dtype, dtype)


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_the_batch_and_the_pages_change_nothing_in_float32(folders, name):
    """The same tokens alone and as one of several in a batch of other lengths, on other pages and slots: the same bits."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    reqs = requests_for(name, [130, 70, 33], seed=43)
    eng = engine_for(folder, "float32")
    alone = run_trace(eng, whole_trace(reqs))
    keep = eng.open()
    eng.step([StepEntry(keep, reqs["r1"][:65], None)])                      # holds a slot and two pages
    s = {r: eng.open() for r in reqs}
    got = eng.step([StepEntry(s[r], reqs[r], "all") for r in ("r2", "r0", "r1")]).float().cpu().numpy()
    assert np.array_equal(got[:33], alone["r2"]) and np.array_equal(got[33:163], alone["r0"])
    assert np.array_equal(got[163:], alone["r1"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_the_second_stream_changes_nothing(folders, name, dtype, monkeypatch):
    """Decode steps with the feed-forward beside the mixer on a second stream and with both in turn on one: the same bits."""
    from exl3_server_b200.engine.decode import DecodeRunner
    reqs = requests_for(name, [80, 33, 5], seed=47)
    steps = batched_trace(reqs, [["r0", "r1", "r2"]], {"r0": 40, "r1": 2, "r2": 1})
    with_side = run_trace(engine_for(folders[name], dtype), steps)
    make = DecodeRunner._batch

    def without(self, *args, **kwargs):
        batch = make(self, *args, **kwargs)
        assert batch.side is not None
        batch.side = None
        return batch
    monkeypatch.setattr(DecodeRunner, "_batch", without)
    alone = run_trace(engine_for(folders[name], dtype), steps)
    for rid in reqs:
        assert np.array_equal(with_side[rid], alone[rid]), rid


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_long_decoding(folders, name, dtype):
    """Three tokens of prompt, then 200 decoded one by one over three page borders and past most windows, two
    sequences side by side."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    reqs = requests_for(name, [203, 180], seed=17)
    pm = plain(folder)
    want = [pm.logits(reqs["r0"]).numpy(), pm.logits(reqs["r1"]).numpy()]
    eng = engine_for(folder, dtype)
    s = [eng.open(), eng.open()]
    got = [[], []]
    out = eng.step([StepEntry(s[0], reqs["r0"][:3], "all"), StepEntry(s[1], reqs["r1"][:3], "all")]).float().cpu().numpy()
    got[0].append(out[:3]); got[1].append(out[3:])
    for i in range(3, 203):
        live = [k for k in (0, 1) if i < len(reqs[f"r{k}"])]
        out = eng.step([StepEntry(s[k], [reqs[f"r{k}"][i]], "all") for k in live]).float().cpu().numpy()
        for j, k in enumerate(live):
            got[k].append(out[j:j + 1])
    for k in (0, 1):
        close_enough(np.concatenate(got[k]), want[k], dtype, k)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_reused_slot_shows_nothing_of_its_former_owner(folders, dtype):
    """A sequence's pages go to the next sequence, which must see none of the old rows, also when it is shorter than the
    old one."""
    from exl3_server_b200 import StepEntry
    folder = folders["mixed"]
    reqs = requests_for("mixed", [190, 30], seed=23)
    want = plain(folder).logits(reqs["r1"]).numpy()
    eng = engine_for(folder, dtype, max_tokens=256)
    for _ in range(3):
        s = eng.open()
        eng.step([StepEntry(s, reqs["r0"], None)])
        eng.close(s)
        s2 = eng.open()
        assert s2 == s
        got = [eng.step([StepEntry(s2, reqs["r1"][:9], "all")]).float().cpu().numpy()]
        for t in reqs["r1"][9:]:
            got.append(eng.step([StepEntry(s2, [t], "all")]).float().cpu().numpy())
        eng.close(s2)
        close_enough(np.concatenate(got), want, dtype, "after reuse")
    eng.cache.check()


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation_through_the_entry_point(folders, name):
    from exl3_server_b200 import GenerateOptions
    folder = folders[name]
    prompts = list(requests_for(name, [5, 70, 1, 33], seed=29).values())
    eng = engine_for(folder, "float32")
    res = eng.generate(prompts, GenerateOptions(max_tokens=24, ignore_eos=True, max_batch=3))
    pm = plain(folder)
    for p, r in zip(prompts, res):
        assert r.tokens == pm.greedy(p, 24)
        assert r.finish_reason == "length"
    assert eng.cache.tokens_held() == 0
    # bfloat16: the same call runs and every token is in range (near-ties may fall the other way)
    eng = engine_for(folder, "bfloat16")
    res = eng.generate(prompts, GenerateOptions(max_tokens=24, ignore_eos=True))
    assert all(len(r.tokens) == 24 and all(0 <= t < CONFIGS[name].vocab for t in r.tokens) for r in res)
    eng.check_kernels()


@pytest.mark.parametrize("name", ["mixed", "odd", "twice"])
def test_residual_stream_layer_by_layer(folders, name):
    """The float32 residual after every layer that runs against the plain implementation's; a layer's last kernel also adds what
    joins the residual ahead of the next one."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    toks = requests_for(name, [75], seed=31)["r0"]
    pm = plain(folder)
    want = list(pm.layers(toks))
    runs = P.layer_runs(pm.cfg)
    for i in range(len(runs) - 1):
        t = runs[i + 1][1]
        if t is not None:
            want[i] = want[i] + pm.w["loop.step"][t] + (pm.w["embed"][torch.tensor(toks)] if t > 0 else 0)
    eng = engine_for(folder, "float32")
    seen = []
    for b in eng.model.blocks:
        def wrapped(stream, *args, f=b.forward, **kwargs):
            f(stream, *args, **kwargs)
            seen.append(stream.h.clone())
        b.forward = wrapped
    s = eng.open()
    eng.step([StepEntry(s, toks, None)])
    assert len(seen) == len(want)
    for i, (a, b) in enumerate(zip(seen, want)):
        assert rel_err(a.cpu().numpy(), b.numpy()) <= TOL["float32"], i


def test_replay_program_and_command_line(folders, tmp_path):
    folder = folders["mixed"]
    vocab = CONFIGS["mixed"].vocab
    reqs = requests_for("mixed", [40, 7], seed=4)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": reqs["r0"][:38], "want": [0, 37]},
                                {"id": "b", "tokens": reqs["r1"][:6], "want": []}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": [reqs["r0"][38]], "want": [0]},
                                {"id": "b", "tokens": [reqs["r1"][6]], "want": [0]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": [reqs["r0"][39]], "want": []}], "end": ["a"]},
        {"step": 3, "entries": [{"id": "b", "tokens": reqs["r1"], "want": [6]}], "end": ["b"]},
    ]
    pm = plain(folder)
    la, lb = pm.logits(reqs["r0"]).numpy(), pm.logits(reqs["r1"]).numpy()
    out = tmp_path / "float32"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                       timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
    s0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, vocab)
    s1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(-1, vocab)
    s3 = np.fromfile(out / "3.f32", dtype="<f4").reshape(-1, vocab)
    assert rel_err(s0, la[[0, 37]]) <= TOL["float32"]
    assert rel_err(s1, np.stack([la[38], lb[6]])) <= TOL["float32"]
    assert rel_err(s3, lb[6:7]) <= TOL["float32"]
    p = subprocess.run([sys.executable, "-m", "exl3_server_b200", "--model", folder, "-p", "5,6,7", "--max-tokens", "5",
                        "--ignore-eos", "--dtype", "float32"], capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.strip() == ",".join(map(str, pm.greedy([5, 6, 7], 5)))
