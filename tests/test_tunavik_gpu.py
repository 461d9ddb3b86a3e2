"""The Tunavik decoder in the engine against the plain implementation (tests/plain_tunavik.py): each mechanism alone, whole
prompts against token-by-token decoding, portions, unequal batches with slots and pages used again, keys far back and at
page borders, every bucket of distances and its edges, first tokens, long decoding, layers that read other layers' keys and
values, generation through the entry point, the replay program; float32 and bfloat16, on configurations that differ in every
size and option.

Routers: a token whose choice between two experts is nearly a tie may choose the other way when its input carries bfloat16
rounding, and then that position's logits differ by far more than rounding.  float32 runs are compared at every position
(requests whose closest decision in the plain implementation is nearer than 1e-4 are drawn again); bfloat16 runs of
configurations with routers may have a share of positions beyond the bound, and the median must be well within it.
"""
import json
import os
import shutil
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import batched_trace, random_requests, rel_err, run_trace, tail_trace, whole_trace
from plain_tunavik import PlainTunavik, bucket
from tunavik_configs import CONFIGS, ROUTED, make_tunavik

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
LENGTHS = {"mixed": [1, 2, 9, 64, 65, 150], "odd": [1, 3, 20, 64, 66, 131], "wide": [3, 17, 63, 128, 129, 300]}
ONLY_LENGTHS = [1, 2, 31, 64, 129, 140]
# bfloat16 with routers: the share of positions that may be beyond the bound (a pick that falls the other way also changes
# what later positions read of this one)
FLIP_SHARE = 0.25
TOL = {"float32": 1e-5, "bfloat16": 5e-2}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("tunavik")
    return {name: make_tunavik(name, str(root / name)) for name in CONFIGS}


_plain = {}


def plain(folder):
    if folder not in _plain:
        _plain[folder] = PlainTunavik(folder)
    return _plain[folder]


def engine_for(folder, dtype, max_tokens=2048):
    from exl3_server_b200 import Engine
    return Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens)


def requests_for(name, folder, lengths, seed):
    """Random requests none of whose routers' decisions is a close call in the plain implementation."""
    pm = plain(folder)
    out = {}
    for i, n in enumerate(lengths):
        for attempt in range(20):
            toks = random_requests(CONFIGS[name].vocab, [n], seed=seed + 1000 * i + 17 * attempt)["r0"]
            if pm.closest_call(toks) >= 1e-4:
                break
        out[f"r{i}"] = toks
    return out


def position_errors(got, want):
    return np.max(np.abs(got.astype(np.float64) - want.astype(np.float64)), axis=1) / max(1e-30, np.max(np.abs(want)))


def close_enough(got, want, dtype, name, what):
    assert got.shape == want.shape, what
    assert np.isfinite(got).all(), what
    err = position_errors(got, want)
    bad = err > TOL[dtype]
    if dtype == "bfloat16" and name in ROUTED:
        assert bad.sum() <= max(1, int(FLIP_SHARE * len(err))) and np.median(err) <= TOL[dtype] / 2, \
            f"{what}: {bad.sum()} of {len(err)} positions beyond the bound, median error {np.median(err):.3e}"
        return
    assert not bad.any(), (f"{what}: differs from the plain implementation by {err.max():.3e} (bound {TOL[dtype]:.0e}); "
                           f"first wrong position {int(np.argmax(bad))} of {len(err)}")


def check(got, want, dtype, name, what):
    assert set(got) == set(want)
    for rid in want:
        close_enough(got[rid], want[rid], dtype, name, f"{what}, request {rid}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in CONFIGS if not n.startswith("random")])
def test_whole_decoded_and_batched(folders, name, dtype):
    folder = folders[name]
    requests = requests_for(name, folder, LENGTHS.get(name, ONLY_LENGTHS), seed=3)
    pm = plain(folder)
    want = {rid: pm.logits(t).numpy() for rid, t in requests.items()}
    eng = engine_for(folder, dtype)
    check(run_trace(eng, whole_trace(requests)), want, dtype, name, "whole")
    check(run_trace(eng, tail_trace(requests, 45)), want, dtype, name, "last 45 one by one")
    # everything but the first token decoded: the prompt path and the one-token path must walk the same sums
    short = {rid: t for rid, t in requests.items() if len(t) <= 70}
    check(run_trace(eng, tail_trace(short, 1000)), {rid: want[rid] for rid in short}, dtype, name, "token by token")
    ids = list(requests)
    # two batches one after the other, so that slots and pages are used again
    batches = [[ids[5], ids[0], ids[2], ids[3]], [ids[1], ids[4], ids[0]]]
    prompt_len = {rid: max(1, len(requests[rid]) - k) for rid, k in zip(ids, (0, 1, 4, 40, 33, 70))}
    check(run_trace(eng, batched_trace(requests, batches, prompt_len)),
          {rid: want[rid] for b in batches for rid in b}, dtype, name, "batched")
    assert eng.cache.tokens_held() == 0
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in CONFIGS if n.startswith("random")])
def test_configurations_drawn_from_a_seed(folders, name, dtype):
    """Layer orders, sizes, counts and constants that nobody chose: whole prompts, the last tokens one by one, and
    a batch of unequal requests decoded together."""
    folder = folders[name]
    requests = requests_for(name, folder, [1, 2, 40, 66, 150], seed=41)
    pm = plain(folder)
    want = {rid: pm.logits(t).numpy() for rid, t in requests.items()}
    eng = engine_for(folder, dtype)
    check(run_trace(eng, whole_trace(requests)), want, dtype, name, "whole")
    check(run_trace(eng, tail_trace(requests, 70)), want, dtype, name, "last 70 one by one")
    ids = list(requests)
    prompt_len = {rid: max(1, len(requests[rid]) - k) for rid, k in zip(ids, (0, 1, 35, 3, 80))}
    check(run_trace(eng, batched_trace(requests, [ids[::-1]], prompt_len)), want, dtype, name, "batched")
    assert eng.cache.tokens_held() == 0
    eng.check_kernels()


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_float32_cuttings_agree_closely(folders, name):
    requests = requests_for(name, folders[name], LENGTHS[name], seed=5)
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
    toks = requests_for(name, folder, [430], seed=9)["r0"]
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
        close_enough(np.concatenate(got), want, dtype, name, f"portions {cuts}")
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_portions_in_one_batch(folders, dtype):
    """Rows that go on by portions of different sizes in the same steps, beside a row that starts."""
    from exl3_server_b200 import StepEntry
    folder = folders["mixed"]
    reqs = requests_for("mixed", folder, [150, 90, 40], seed=13)
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
        close_enough(np.concatenate(got[r]), want[r], dtype, "mixed", r)


def _rewrite(src, folder, change):
    os.makedirs(folder)
    shutil.copy(os.path.join(src, "config.json"), folder)
    from safetensors import safe_open
    from exl3_server_b200.weights.safetensors_io import write_safetensors
    with safe_open(os.path.join(src, "model.safetensors"), framework="pt") as f:
        tensors = {k: f.get_tensor(k).float() for k in f.keys()}
    change(tensors)
    write_safetensors(os.path.join(folder, "model.safetensors"), ((k, v.to(torch.bfloat16)) for k, v in tensors.items()),
                      metadata={"format": "pt"})


MARKED = 77


def _mark_features(t):
    """The last feature of the model is about one for every token wherever it stands (its sinusoid is a cosine of the lowest
    frequency), the one before it is on for the marked token only (a sine that stays below a tenth for the positions here)."""
    t["embed"][:, -2:] = 0.0
    t["embed"][MARKED, -2] = 6.0
    t["embed.norm"][-2:] = 0.0


def _marked_attention(src, folder, layers):
    """A copy of a model in which one token's key stands out for every query of the attention of ``layers`` (pairs of the
    layer that asks and the layer whose keys it reads): the query matrix sends the last feature, and the key matrix the one
    before it, to the same features of every head, so that the marked key's score is far above the others' whatever the
    distance adds."""
    def change(t):
        _mark_features(t)
        for asks, keys in layers:
            for name, col in ((f"l{asks}.mix.q", -1), (f"l{keys}.mix.k", -2)):
                t[name][:, col] = 3.0
                t[name + ".b"][:] = 0.0
            t[f"l{keys}.mix.v"][:, -2] = 1.0          # and its value is several times the others'
            t[f"l{asks}.mix.rel"] *= 0.5
    _rewrite(src, folder, change)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, layers", [("only_attention", [(0, 0)]), ("only_tiles", [(0, 0)]), ("only_reader", [(1, 0)])])
def test_a_key_that_stands_out(folders, tmp_path, name, layers, dtype):
    """The marked key sits first, second, on both sides of page borders, hundreds of tokens back and among the last; losing it
    or reading a neighbour instead changes the logits by far more than the bound.  Whole prompts, and the last 95 tokens
    decoded one by one; for a layer that reads another layer's keys too."""
    folder = str(tmp_path / "m")
    _marked_attention(folders[name], folder, layers)
    pm = PlainTunavik(folder)
    base = [t if t != MARKED else 5 for t in random_requests(CONFIGS[name].vocab, [700], seed=21)["r0"]]
    plainly = pm.logits(base).numpy()
    eng = engine_for(folder, dtype)
    for place in [0, 1, 63, 64, 127, 128, 300, 639, 640, 698]:
        toks = list(base)
        toks[place] = MARKED
        want = pm.logits(toks).numpy()
        assert rel_err(plainly[-1:], want[-1:]) > 0.15, place            # the last query sees the key
        got = run_trace(eng, whole_trace({"a": toks}))["a"]
        assert rel_err(got, want) <= TOL[dtype], ("whole", place)
        got = run_trace(eng, tail_trace({"a": toks}, 95))["a"]
        assert rel_err(got, want) <= TOL[dtype], ("decoded", place)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_attention", "only_tiles"])
@pytest.mark.parametrize("rows, limit", [(8, 64), (9, 80), (16, 300)])
def test_every_bucket_of_distances_alone(folders, tmp_path, name, rows, limit, dtype):
    """A table that lifts one bucket far above the others, for single-distance buckets, the first and the later geometric
    ones and the last (everything farther); 8 rows up to 64 put the buckets' edges on exact powers.  A bucket that starts or
    ends one distance off changes the logits by far more than the bound."""
    folder = str(tmp_path / "m")
    heads = CONFIGS[name].layers[0].mixer["heads"]

    def change(t):
        t["l0.mix.rel"] = torch.zeros(rows, heads)
        t["l0.mix.v"] *= 4.0
    _rewrite(folders[name], folder, change)
    cfg = json.load(open(os.path.join(folder, "config.json")))
    cfg["layers"][0]["mixer"]["bias_max"] = limit
    json.dump(cfg, open(os.path.join(folder, "config.json"), "w"))
    pm = PlainTunavik(folder)
    toks = random_requests(128, [330], seed=37)["r0"]
    flat = pm.logits(toks).numpy()
    half = rows // 2
    for b in sorted({0, 1, half - 1, half, half + 1, rows - 2, rows - 1}):
        lifted = str(tmp_path / f"b{b}")

        def lift(t):
            t["l0.mix.rel"][b] = torch.tensor([7.0, 6.0, 7.5, 6.5][:heads])
        _rewrite(folder, lifted, lift)
        pl = PlainTunavik(lifted)
        want = pl.logits(toks).numpy()
        seen = [p for p in range(330) if any(bucket(n, rows, limit) == b for n in range(p + 1))]
        assert rel_err(flat[seen], want[seen]) > 0.1, b
        eng = engine_for(lifted, dtype)
        assert rel_err(run_trace(eng, whole_trace({"a": toks}))["a"], want) <= TOL[dtype], ("whole", b)
        assert rel_err(run_trace(eng, tail_trace({"a": toks}, 150))["a"], want) <= TOL[dtype], ("decoded", b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_attention", "only_tiles"])
def test_the_sink_counts(folders, tmp_path, name, dtype):
    """Sinks far above the scores: leaving the sink out, scaling it or giving it a bias would change every row; with a far
    bucket that is far from zero, which the kernels fold into the sink."""
    folder = str(tmp_path / "m")

    def change(t):
        t["l0.mix.sink"][:] = torch.tensor([6.0, 5.0, 7.0, 4.0])
        t["l0.mix.rel"][-1] = torch.tensor([3.0, -2.0, 2.5, 4.0])
    _rewrite(folders[name], folder, change)
    pm = PlainTunavik(folder)
    toks = random_requests(128, [200], seed=33)["r0"]
    want = pm.logits(toks).numpy()
    assert rel_err(plain(folders[name]).logits(toks).numpy(), want) > 0.05
    eng = engine_for(folder, dtype)
    assert rel_err(run_trace(eng, whole_trace({"a": toks}))["a"], want) <= TOL[dtype]
    assert rel_err(run_trace(eng, tail_trace({"a": toks}, 90))["a"], want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_temperature_steps_where_it_should(folders, tmp_path, dtype):
    """A temperature that multiplies every few positions: a step one position off shows at that position."""
    folder = str(tmp_path / "m")
    _rewrite(folders["only_attention"], folder, lambda t: None)
    path = os.path.join(folder, "config.json")
    cfg = json.load(open(path))
    toks = random_requests(128, [140], seed=35)["r0"]
    eng = None
    for every in (1, 7, 64):
        cfg["layers"][0]["mixer"]["q_temp"] = {"coef": 1.5, "every": every}
        json.dump(cfg, open(path, "w"))
        want = PlainTunavik(folder).logits(toks).numpy()
        late = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], q_temp={"coef": 1.5, "every": every + 1}))])
        other = PlainTunavik(folder)
        other.cfg = late
        assert rel_err(other.logits(toks).numpy()[every - 1:every], want[every - 1:every]) > 1e-3 or every == 1
        eng = engine_for(folder, dtype)
        assert rel_err(run_trace(eng, whole_trace({"a": toks}))["a"], want) <= TOL[dtype], every
        assert rel_err(run_trace(eng, tail_trace({"a": toks}, 70))["a"], want) <= TOL[dtype], every


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_the_batch_and_the_pages_change_nothing_in_float32(folders, name):
    """The same tokens alone and as one of several in a batch of other lengths, on other pages and slots: the same bits."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    reqs = requests_for(name, folder, [130, 70, 33], seed=43)
    eng = engine_for(folder, "float32")
    alone = run_trace(eng, whole_trace(reqs))
    keep = eng.open()
    eng.step([StepEntry(keep, reqs["r1"][:65], None)])                      # holds a slot and two pages
    s = {r: eng.open() for r in reqs}
    got = eng.step([StepEntry(s[r], reqs[r], "all") for r in ("r2", "r0", "r1")]).float().cpu().numpy()
    assert np.array_equal(got[:33], alone["r2"]) and np.array_equal(got[33:163], alone["r0"])
    assert np.array_equal(got[163:], alone["r1"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_long_decoding(folders, name, dtype):
    """Three tokens of prompt, then 200 decoded one by one over three page borders and past every table's reach, two
    sequences side by side."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    reqs = requests_for(name, folder, [203, 180], seed=17)
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
        close_enough(np.concatenate(got[k]), want[k], dtype, name, k)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_reused_slot_shows_nothing_of_its_former_owner(folders, dtype):
    """A sequence's pages go to the next sequence, which must see none of the old rows, also when it is shorter than the
    old one."""
    from exl3_server_b200 import StepEntry
    folder = folders["mixed"]
    reqs = requests_for("mixed", folder, [190, 30], seed=23)
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
        close_enough(np.concatenate(got), want, dtype, "mixed", "after reuse")
    eng.cache.check()


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation_through_the_entry_point(folders, name):
    from exl3_server_b200 import GenerateOptions
    folder = folders[name]
    prompts = list(requests_for(name, folder, [5, 70, 1, 33], seed=29).values())
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


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_residual_stream_layer_by_layer(folders, name):
    """The float32 residual after every layer against the plain implementation's."""
    from exl3_server_b200 import StepEntry
    folder = folders[name]
    toks = requests_for(name, folder, [75], seed=31)["r0"]
    want = plain(folder).layers(toks)
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
    reqs = requests_for("mixed", folder, [40, 7], seed=4)
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
