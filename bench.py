#!/usr/bin/env python3
"""Decode and prefill throughput of the engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

The default run has the layer sizes of the 2B-class MiniCPM configuration (40
layers, width 2304, 36/36 heads of 64, feed-forward 5760, vocabulary 122753,
tied head) with random bfloat16 weights N(0, 0.02), a batch of 8 and a context
of 4096 tokens.  A "step" is one decode step of the whole batch.  It prints ONE
JSON line: ``value`` is decoded tokens per second timed on the device over K
steps (CUDA events), ``e2e`` the same through ``Engine.generate`` with host
token ids in and out every step, ``prefill`` one 2,048-token prompt,
``roofline`` the decode step's bytes (every weight once plus the live cache)
over its time, ``points`` decode at batch 1 and 64 and, unless ``--no-points``,
the other measurements the baseline names: the 2B sizes at contexts of 128 and
2,048 tokens, the 8B-class MiniCPM4 sizes (32 query heads on 2 key/value heads
of 128; decode at batch 1, 8, 64 and a 2,048-token prefill) and the 0.5B-class
MiniCPM4 sizes (64 prompts of 16 to 2,048 tokens in one prefill step, then 256
decode steps); ``points_frac`` gives each point's fraction of its roofline
(HBM bytes for decode, bfloat16 flops for prefill).  Every repeat of a point is
printed to stderr as it is measured; a point's value is its best repeat.
Peaks come from MEASURED_PEAKS.json when it exists, else from the stated
fallback.

``--only decode|prefill|unequal`` with ``--sizes NAME`` runs one part at any of
the size tables and prints a short JSON line (for profiling small cases).

``--only designs`` measures the Rigitar decoder (latent attention, minGRU and
dense xIELU layers) and the Nikodra decoder (attention with a sink, attention in
blocks beside retention, wkv recurrences, dense GELU layers) and the Nibelix
decoder (lightning recurrences, differential attention over a window, dense and
routed feed-forwards) and the Potodra decoder (a residual of four streams, attention over a window that keeps the first
keys, matrix memories with exponential gates, a gated delta rule beside causal attention, dense and routed
feed-forwards) and the Tunavik decoder (causal attention with distance biases, a sink and shared keys and values, routed
feed-forwards) and the Soporax decoder (latent attention, attention over a window and causal attention with gates, each beside
its feed-forward on one norm, experts from a table, layers that run twice) beside the Llama-family decoder at equal width, depth, head count and feed-forward width,
with random weights: one prompt of
``--prefill-tokens`` tokens and decode steps at ``--batch`` and ``--context``,
for each of the size pairs in ``DESIGN_SIZES`` (or the one named by
``--design-sizes``); ``--design-arch`` runs one of the designs only (for profiling).

Only one GPU is supported: for N > 1 it says so and exits with 2.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

FALLBACK_HBM_GBS = 6650.0
FALLBACK_BF16_TFLOPS = 1590.0
HEADLINE = "minicpm-2b"


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    hbm, tf, src = FALLBACK_HBM_GBS, FALLBACK_BF16_TFLOPS, "fallback"
    if os.path.exists(path):
        try:
            with open(path) as f:
                j = json.load(f)
            hbm = float(j.get("hbm_gbs", hbm))
            tf = float(j.get("bf16_tflops", tf))
            src = "measured"
        except (OSError, ValueError):
            pass
    return hbm, tf, src


def say(msg: str) -> None:
    print(f"[bench] {msg}", file=sys.stderr, flush=True)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""

    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            out, _ = self.proc.communicate(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
            out, _ = self.proc.communicate()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in out.splitlines():
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 6:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for n, v in zip(names, parts[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm)}


# Size pairs for ``--only designs``: width, layers, heads, feed-forward width, vocabulary; the Llama side has heads of
# ``head_dim`` on ``kv_heads`` key/value heads; the Rigitar side has latent attention with these sizes in half of its
# layers (every second of them reading the rows of the one before), minGRU of the model's width in the others, and
# the dense feed-forward in all; the Nikodra side repeats attention, attention, attention in blocks of 1,024 positions
# beside retention (states of 64 x head_dim), wkv (heads of 64), with the dense feed-forward in all.
DESIGN_SIZES = {
    "w2048": dict(width=2048, layers=8, heads=16, ff=5632, vocab=32000, head_dim=128, kv_heads=16,
                  latent=dict(dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512)),
    "w4096": dict(width=4096, layers=4, heads=32, ff=11008, vocab=32000, head_dim=128, kv_heads=8,
                  latent=dict(dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512)),
}


def nikodra_config(z):
    from exl3_server_b200.config.nikodra import NikodraConfig, NikodraLayer
    hd = z["head_dim"]
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5, "v_mix": True,
           "rot": {"base": 500000.0, "dims": hd, "scaling": {"factor": 8.0, "original": 4096, "fast": 16.0, "slow": 2.0}}}
    left = {k: att[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")}
    left["mask"] = {"size": 1024}
    right = {"heads": z["heads"], "dim": 64, "vdim": hd, "decay": [1.0 - 2.0 ** (-4.0 - 6.0 * i / z["heads"]) for i in range(z["heads"])],
             "rot": {"base": 10000.0, "dims": 64}}
    mlp = {"kind": "dense", "ff": z["ff"]}
    kinds = [("attention", att), ("attention", att), ("parallel", {"left": left, "right": right}),
             ("wkv", {"heads": z["width"] // 64, "dim": 64, "decay_rank": 64})]
    layers = [NikodraLayer(kinds[i % 4][0], dict(kinds[i % 4][1]), dict(mlp)) for i in range(z["layers"])]
    return NikodraConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, residual_mult=0.5,
                         bigram={"buckets": 65521, "mul_prev": 1000003, "mul_cur": 31}, layers=layers)


def nibelix_config(z):
    """Nibelix at one of the size pairs: layers repeat lightning + dense, attention + routed, lightning + routed,
    attention + dense.  Lightning states are 64 x head_dim (the Nikodra side's retention has the same); the two maps
    of a differential head have head_dim / 2 features each, so a key row is as wide as the other sides' keys, over a
    window of 1,024 positions; 14 experts and 2 identity outputs in 4 groups of which 2 are kept, 2 picks a token,
    experts and the shared expert a quarter of the dense feed-forward's width."""
    from exl3_server_b200.config.nibelix import NibelixConfig, NibelixLayer
    hd = z["head_dim"]
    lightning = {"heads": z["heads"], "dim": 64, "vdim": hd,
                 "decay": [1.0 - 2.0 ** (-4.0 - 6.0 * i / z["heads"]) for i in range(z["heads"])]}
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": hd // 2, "vdim": hd, "scale": (hd // 2) ** -0.5,
           "diff": 0.35, "mask": {"size": 1024}, "rot": {"base": 500000.0, "dims": hd // 2}}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "shared": {"ff": z["ff"] // 4},
           "router": {"experts": 14, "identity": 2, "top": 2, "scale": 1.5, "groups": {"count": 4, "keep": 2}}}
    kinds = [("lightning", lightning, dense), ("attention", att, moe), ("lightning", lightning, moe),
             ("attention", att, dense)]
    layers = [NibelixLayer(kinds[i % 4][0], dict(kinds[i % 4][1]), dict(kinds[i % 4][2])) for i in range(z["layers"])]
    return NibelixConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, residual_mult=0.5, logit_softcap=30.0,
                         layers=layers)


def potodra_config(z):
    """Potodra at one of the size pairs: four streams; layers repeat attention + routed, matrix memory with exponential
    gates + dense, causal attention beside a gated delta rule + dense, matrix memory + routed.  The attention layers have
    the other sides' heads over a window of 1,024 positions that keeps the first 64 keys, capped scores and a sink per
    head; the causal attention has the same heads; the recurrences' states are 64 x head_dim per head (the Nikodra and
    Nibelix sides' recurrences have the same), the delta rule with convolutions of 4 taps; 16 experts in 4 groups of
    which 2 are kept, 2 picks a token, experts and the shared expert a quarter of the dense feed-forward's width."""
    from exl3_server_b200.config.potodra import PotodraConfig, PotodraLayer
    hd = z["head_dim"]
    plain = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5,
             "rot": {"base": 500000.0, "dims": hd}, "softcap": None, "mask": None}
    att = dict(plain, softcap=30.0, mask={"size": 1024, "keep_first": 64})
    memory = {"heads": z["heads"], "dim": 64, "vdim": hd, "gate_cap": 12.0}
    delta = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": 64, "vdim": hd, "conv": 4}
    par = {"left": plain, "right": delta, "left_scale": 0.7, "right_scale": 0.4}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4, "limit": 7.0}, "shared": {"ff": z["ff"] // 4, "limit": 7.0},
           "router": {"experts": 16, "top": 2, "groups": {"count": 4, "keep": 2}}}
    kinds = [("attention", att, moe), ("mlstm", memory, dense), ("parallel", par, dense), ("mlstm", memory, moe)]
    layers = [PotodraLayer(kinds[i % 4][0], dict(kinds[i % 4][1]), dict(kinds[i % 4][2])) for i in range(z["layers"])]
    return PotodraConfig(vocab=z["vocab"], width=z["width"], streams=4, norm_eps=1e-6, embedding_scale=2.0, layers=layers)


def tunavik_config(z):
    """Tunavik at one of the size pairs: every layer has the other sides' attention heads (causal, a bias for keys less than
    256 positions back, a sink, one norm over all heads) and a routed feed-forward like the Nibelix and Potodra sides': 16
    experts, 2 picks a token, experts and the shared expert a quarter of the dense feed-forward's width.  Every fourth layer
    reads the keys and values of the one before."""
    from exl3_server_b200.config.tunavik import TunavikConfig, TunavikLayer
    hd = z["head_dim"]
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5, "bias_max": 256,
           "q_temp": {"coef": 0.1, "every": 2048}, "kv_from": None}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": 16, "top": 2}, "shared": {"ff": z["ff"] // 4}}
    layers = [TunavikLayer("attention", dict(att, kv_from=i - 1 if i % 4 == 3 else None), dict(moe)) for i in range(z["layers"])]
    return TunavikConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, logit_scale=1.5, logit_softcap=30.0, layers=layers)


def soporax_config(z):
    """Soporax at one of the size pairs: as many layer runs as the other sides have layers, a quarter of them a second pass
    over the same layers.  Layers repeat latent attention (the Rigitar side's sizes, a gate per output feature) + dense,
    attention over a window of 1,024 positions with a sink + routed, causal attention with a gate per head + routed (both
    with the other sides' heads); 16 experts, 2 a token from a table, gated, a quarter of the dense feed-forward's width."""
    from exl3_server_b200.config.soporax import SoporaxConfig, SoporaxLayer
    hd, lat = z["head_dim"], z["latent"]
    heads = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5}
    kinds = [
        ("latent_attention", dict(heads=z["heads"], scale=(lat["dim"] + lat["rot_dim"]) ** -0.5,
                                  rot={"base": 10000.0, "dims": lat["rot_dim"],
                                       "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}, **lat),
         {"kind": "dense", "ff": z["ff"], "limit": 7.0}),
        ("attention", dict(heads, mask={"size": 1024}), None),
        ("attention_2", dict(heads, rot={"base": 500000.0, "dims": hd,
                                         "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}), None)]
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": 16, "top": 2}}
    twice = z["layers"] // 4
    layers = [SoporaxLayer(k, dict(m), dict(f or moe)) for k, m, f in (kinds[i % 3] for i in range(z["layers"] - twice))]
    return SoporaxConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, logit_scale=0.5,
                         loop={"start": 1, "stop": 1 + twice, "times": 2}, layers=layers)


def design_configs(name: str):
    """(Rigitar configuration, Llama configuration) of one size pair."""
    import exl3_server_b200 as E
    from exl3_server_b200.config.rigitar import RigitarConfig, RigitarLayer
    z = DESIGN_SIZES[name]
    lat = z["latent"]
    layers = []
    for i in range(z["layers"]):
        mlp = {"kind": "dense", "ff": z["ff"]}
        if i % 4 in (1, 2):
            m = dict(heads=z["heads"], scale=(lat["dim"] + lat["rot_dim"]) ** -0.5,
                     rot={"base": 10000.0, "dims": lat["rot_dim"]}, **lat)
            if i % 4 == 2:
                m["kv_from"] = i - 1
            layers.append(RigitarLayer("latent_attention", m, mlp))
        else:
            layers.append(RigitarLayer("mingru", {"width": z["width"]}, mlp))
    rig = RigitarConfig(vocab=z["vocab"], width=z["width"], norm_eps=1e-6, layers=layers)
    llama = E.LlamaConfig(hidden_size=z["width"], num_hidden_layers=z["layers"], num_attention_heads=z["heads"],
                          num_key_value_heads=z["kv_heads"], head_dim=z["head_dim"], intermediate_size=z["ff"],
                          vocab_size=z["vocab"], tie_word_embeddings=False, max_position_embeddings=0)
    return rig, llama


class Rig:
    """A random-weight model of one of the size tables with a cache, and the timed pieces."""

    @classmethod
    def of_config(cls, name: str, cfg, cache_tokens: int, max_slots: int) -> "Rig":
        """The same for any registered architecture's typed configuration."""
        import torch
        import exl3_server_b200 as E
        from exl3_server_b200.config.registry import resolve_architecture
        from exl3_server_b200.engine.model import Model, plan_manifest
        from exl3_server_b200.weights.random_init import random_tensors
        self = cls.__new__(cls)
        self.torch, self.E, self.name, self.cfg = torch, E, name, cfg
        dev = torch.device("cuda:0")
        t0 = time.time()
        plan = resolve_architecture(cfg.to_dict()).build_plan(cfg)
        self.layers = self.layers_full = len(plan.layers)
        self.vocab = plan.head.vocab
        tensors = dict(random_tensors(plan_manifest(plan), seed=0, std=0.02, norm_std=None, dtype=torch.bfloat16,
                                      device=dev))
        self.model = Model(plan, tensors, torch.bfloat16, dev)
        del tensors
        self.engine = E.Engine(self.model, max_tokens=cache_tokens, max_slots=max_slots)
        self.gen = torch.Generator().manual_seed(1)
        say(f"{name}: {self.layers} layers, cache of {cache_tokens} tokens, ready in {time.time() - t0:.1f}s")
        return self

    def __init__(self, sizes_name: str, layers: int, cache_tokens: int, max_slots: int):
        import torch
        import exl3_server_b200 as E
        from exl3_server_b200.config.presets import SIZES, sizes
        from exl3_server_b200.engine.model import Model, plan_manifest
        from exl3_server_b200.models.llama import build_plan
        from exl3_server_b200.weights.random_init import random_tensors
        self.torch, self.E = torch, E
        self.name = sizes_name
        self.layers_full = SIZES[sizes_name]["num_hidden_layers"]
        self.layers = min(layers, self.layers_full) if layers > 0 else self.layers_full
        # the residual scale belongs to the full model whatever the number of layers run
        self.cfg = E.LlamaConfig(**sizes(sizes_name, num_hidden_layers=self.layers))
        self.vocab = self.cfg.vocab_size
        dev = torch.device("cuda:0")
        t0 = time.time()
        plan = build_plan(self.cfg)
        tensors = dict(random_tensors(plan_manifest(plan), seed=0, std=0.02, norm_std=None, dtype=torch.bfloat16,
                                      device=dev))
        self.model = Model(plan, tensors, torch.bfloat16, dev)
        del tensors
        self.engine = E.Engine(self.model, max_tokens=cache_tokens, max_slots=max_slots)
        self.gen = torch.Generator().manual_seed(1)
        say(f"{sizes_name}: {self.layers} of {self.layers_full} layers, cache of {cache_tokens} tokens, ready in "
            f"{time.time() - t0:.1f}s")

    def close(self):
        self.engine = self.model = None
        gc.collect()
        self.torch.cuda.empty_cache()

    def prompts(self, n, length):
        return [self.torch.randint(0, self.vocab, (length,), generator=self.gen).tolist() for _ in range(n)]

    def kv_bytes_per_token(self):
        return sum(g.bytes_per_token(2) for g in self.engine.cache.groups)

    def context_bytes(self, ctx):
        """Bytes of cache and state that one sequence's decode step at ``ctx`` tokens of context has to move: the
        keys and values it may see (a window or a block of positions bounds them) and its per-sequence state, read
        and written."""
        n = 0
        for g in self.engine.cache.groups:
            seen = ctx
            if g.request.window > 0:
                seen = min(seen, g.request.window)
            if g.request.chunk > 0:
                seen = min(seen, (ctx - 1) % g.request.chunk + 1)
            n += g.bytes_per_token(2) * seen
        for t in self.engine.cache.state.values():
            for part in (t if isinstance(t, tuple) else (t,)):
                n += 2 * part[0].numel() * part.element_size()
        return n

    def prefill_flops(self, lengths):
        """Matrix products of every layer for all tokens, causal attention, the head on one row per prompt."""
        c = self.cfg
        lin = sum(b.mixer.qkv.weight.numel() + b.mixer.o.weight.numel() + b.feed_forward.gate_up.weight.numel()
                  + b.feed_forward.down.weight.numel() for b in self.model.blocks)
        att = sum(2.0 * c.num_attention_heads * c.head_dim * n * n for n in lengths) * self.layers
        return 2.0 * sum(lengths) * lin + att + 2.0 * c.vocab_size * c.hidden_size * len(lengths)

    def fill(self, slots, toks, chunk=8192):
        """Real prefill through the step function, in steps of about ``chunk`` tokens."""
        E = self.E
        per = max(1, chunk // len(slots))
        for a in range(0, len(toks[0]), per):
            self.engine.step([E.StepEntry(s, t[a:a + per], None) for s, t in zip(slots, toks)])

    def decode(self, batch, ctx, steps, warmup):
        """Device time of ``steps`` decode steps that end at ``ctx`` tokens of context: (ms, launches, cache bytes
        read per step)."""
        from exl3_server_b200.engine.decode import DecodeSession
        from exl3_server_b200.ops import kernels as K
        torch, eng = self.torch, self.engine
        ctx0 = max(1, ctx - steps - warmup)
        slots = [eng.open() for _ in range(batch)]
        self.fill(slots, self.prompts(batch, ctx0))
        sess = DecodeSession(eng, slots, [1] * batch)
        for _ in range(warmup):
            sess.step()
        torch.cuda.synchronize()
        l0 = K.launch_count()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(steps):
            sess.step()
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1)
        launches = sess.launches_per_step * steps if sess.launches_per_step else K.launch_count() - l0
        kv = self.kv_bytes_per_token() * batch * (ctx0 + warmup + steps / 2.0)
        sess.close()
        for s in slots:
            eng.close(s)
        return ms, launches, kv

    def decode_point(self, name, batch, ctx, steps, warmup, hbm_gbs, repeats=2):
        """(tokens per second, fraction of the HBM roofline) of the best of ``repeats`` runs; each is printed."""
        best = None
        for r in range(repeats):
            ms, _, kv = self.decode(batch, ctx, steps, warmup)
            rate = batch * steps / (ms / 1e3)
            gbs = (self.model.weight_bytes() + kv) / (ms / steps / 1e3) / 1e9
            say(f"{name} repeat {r}: {ms / steps:.3f} ms/step, {rate:.0f} tok/s, {gbs:.0f} GB/s")
            if best is None or rate > best[0]:
                best = (rate, gbs / hbm_gbs)
        return best

    def prefill(self, tokens, repeats=4, warm=3):
        """Milliseconds of one step with one prompt of ``tokens`` tokens (best repeat; each is printed).  Every
        other timed step starts after a quarter of a second of idling: back to back the steps of the larger sizes
        run into the power cap and each is slower than the one before, after idling the clocks of the smaller
        sizes' short step have to come up again; the burst rate they are compared with was measured on a kernel
        in isolation."""
        torch, E, eng = self.torch, self.E, self.engine
        toks = self.prompts(1, tokens)[0]
        times = []
        for i in range(warm + repeats):
            s = eng.open()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            if i >= warm and (i - warm) % 2 == 1:
                time.sleep(0.25)
            e0.record()
            eng.step([E.StepEntry(s, toks, "last")])
            e1.record()
            torch.cuda.synchronize()
            eng.close(s)
            if i >= warm:
                times.append(e0.elapsed_time(e1))
                say(f"{self.name} prefill of {tokens} tokens, repeat {i - warm}: {times[-1]:.3f} ms")
        return min(times)

    def unequal(self, n_prompts, lo, hi, decode_steps, repeats=2):
        """``n_prompts`` prompts of ``lo`` to ``hi`` tokens (seeded) in ONE prefill step, then ``decode_steps``
        steps of all of them: (prefill tokens, prefill ms, decode ms per step, cache bytes per decode step)."""
        from exl3_server_b200.engine.decode import DecodeSession
        torch, E, eng = self.torch, self.E, self.engine
        lens = torch.randint(lo, hi + 1, (n_prompts,), generator=self.gen).tolist()
        toks = [self.prompts(1, n)[0] for n in lens]
        best_pf, best_dec = None, None
        for r in range(repeats + 1):
            slots = [eng.open() for _ in range(n_prompts)]
            e0, e1, e2 = (torch.cuda.Event(enable_timing=True) for _ in range(3))
            torch.cuda.synchronize()
            e0.record()
            eng.step([E.StepEntry(s, t, "last") for s, t in zip(slots, toks)])
            e1.record()
            sess = DecodeSession(eng, slots, [1] * n_prompts, max_new=decode_steps + 8)
            for _ in range(3):
                sess.step()
            torch.cuda.synchronize()
            e1b = torch.cuda.Event(enable_timing=True)
            e1b.record()
            for _ in range(decode_steps):
                sess.step()
            e2.record()
            torch.cuda.synchronize()
            pf, dec = e0.elapsed_time(e1), e1b.elapsed_time(e2) / decode_steps
            sess.close()
            for s in slots:
                eng.close(s)
            if r == 0:
                continue                                    # records the graphs and warms the kernels
            say(f"{self.name} unequal batch of {n_prompts} ({sum(lens)} tokens), repeat {r - 1}: prefill {pf:.2f} ms, "
                f"decode {dec:.3f} ms/step")
            best_pf = pf if best_pf is None else min(best_pf, pf)
            best_dec = dec if best_dec is None else min(best_dec, dec)
        kv = self.kv_bytes_per_token() * (sum(lens) + n_prompts * (3 + decode_steps / 2.0))
        return lens, best_pf, best_dec, kv


def designs(args) -> int:
    """``--only designs``: prefill and decode throughput of the Rigitar, Nikodra, Nibelix, Potodra, Tunavik and Soporax decoders beside
    the Llama-family decoder of equal sizes; one JSON line."""
    import torch
    torch.cuda.set_device(0)
    hbm_gbs, bf16_tf, peak_src = peaks()
    B, C, T = args.batch, args.context, args.prefill_tokens
    steps, warm = args.steps, max(3, args.warmup)
    page = 64
    room = (B + 1) * ((max(C, T) + page - 1) // page * page + page)
    out = {"only": "designs", "batch": B, "context": C, "prefill_tokens": T, "steps": steps, "dtype": "bf16",
           "data": "synthetic: random weights N(0,0.02), uniform random token ids", "peaks": peak_src, "sizes": {}}
    for name in ([args.design_sizes] if args.design_sizes else sorted(DESIGN_SIZES)):
        rig_cfg, llama_cfg = design_configs(name)
        rec = {}
        for arch, cfg in (("soporax", soporax_config(DESIGN_SIZES[name])), ("tunavik", tunavik_config(DESIGN_SIZES[name])), ("potodra", potodra_config(DESIGN_SIZES[name])), ("nibelix", nibelix_config(DESIGN_SIZES[name])),
                          ("nikodra", nikodra_config(DESIGN_SIZES[name])),
                          ("rigitar", rig_cfg), ("llama", llama_cfg)):
            if args.design_arch not in ("both", arch):
                continue
            rig = Rig.of_config(f"{name}/{arch}", cfg, room, B + 1)
            r = {"weight_bytes": rig.model.weight_bytes(), "cache_bytes_per_token": rig.kv_bytes_per_token()}
            if args.design_part in ("both", "prefill"):
                ms = rig.prefill(T, repeats=2)
                r.update(prefill_ms=ms, prefill_tok_s=T / (ms / 1e3))
            if args.design_part in ("both", "decode"):
                ms, launches, kv = rig.decode(B, C, steps, warm)
                kv = B * rig.context_bytes(C - steps // 2)
                step_weights = rig.model.weight_bytes(B)      # of routed experts, the ones a step of B tokens picks
                gbs = (step_weights + kv) / (ms / steps / 1e3) / 1e9
                r.update(decode_weight_bytes=step_weights, decode_ms_per_step=ms / steps,
                         decode_tok_s=B * steps / (ms / 1e3), decode_gb_s=gbs, decode_hbm_frac=gbs / hbm_gbs,
                         gpu_launches_per_step=int(launches) // steps)
            rec[arch] = r
            rig.close()
        out["sizes"][name] = rec
    print(json.dumps(out))
    return 0


def main() -> int:
    from exl3_server_b200.config.presets import SIZES
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers of the same sizes (stated in config); 0: all")
    ap.add_argument("--prefill-tokens", type=int, default=2048)
    ap.add_argument("--no-points", action="store_true", help="skip everything but the headline measurements")
    ap.add_argument("--sizes", choices=sorted(SIZES), default=HEADLINE,
                    help="layer sizes; other than the default only with --only (a short JSON line)")
    ap.add_argument("--only", choices=["all", "decode", "prefill", "unequal", "designs"], default="all",
                    help="run one part only (for profiling small cases); prints a short JSON line")
    ap.add_argument("--design-sizes", choices=sorted(DESIGN_SIZES), default=None,
                    help="with --only designs: one size pair instead of all")
    ap.add_argument("--design-arch", choices=["both", "soporax", "tunavik", "potodra", "nibelix", "nikodra", "rigitar", "llama"], default="both",
                    help="with --only designs: one of the designs only (both: all of them)")
    ap.add_argument("--design-part", choices=["both", "prefill", "decode"], default="both",
                    help="with --only designs: one of the two measurements only")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference is a C++/CMake program on Apple's MLX and Metal; pip finds nothing to "
                          "install (no setup.py or pyproject.toml) and MLX does not exist for this machine"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.only == "designs":
        return designs(args)
    if args.sizes != HEADLINE and args.only == "all":
        print(f"bench.py: --sizes other than {HEADLINE} needs --only decode, prefill or unequal")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch
    torch.cuda.set_device(0)
    hbm_gbs, bf16_tf, peak_src = peaks()
    B, C, Kst, W = args.batch, args.context, args.steps, args.warmup
    page = 64

    def room(batch, ctx):
        return (batch + 1) * ((ctx + page - 1) // page * page + page)

    # ---- one part only -----------------------------------------------------------------------------------------
    if args.only == "decode":
        rig = Rig(args.sizes, args.layers, room(B, C), B + 1)
        ms, launches, kv = rig.decode(B, C, Kst, W)
        gbs = (rig.model.weight_bytes() + kv) / (ms / Kst / 1e3) / 1e9
        print(json.dumps({"only": "decode", "sizes": args.sizes, "batch": B, "context": C, "layers": rig.layers,
                          "ms_per_step": ms / Kst, "tok_s": B * Kst / (ms / 1e3), "gb_s": gbs,
                          "hbm_frac": gbs / hbm_gbs, "gpu_launches": int(launches)}))
        return 0
    if args.only == "prefill":
        rig = Rig(args.sizes, args.layers, room(1, args.prefill_tokens), 2)
        ms = rig.prefill(args.prefill_tokens, repeats=max(1, Kst // 16))
        tf = rig.prefill_flops([args.prefill_tokens]) / (ms / 1e3) / 1e12
        print(json.dumps({"only": "prefill", "sizes": args.sizes, "tokens": args.prefill_tokens, "layers": rig.layers,
                          "ms": ms, "tok_s": args.prefill_tokens / (ms / 1e3), "tflops": tf, "frac": tf / bf16_tf}))
        return 0
    if args.only == "unequal":
        rig = Rig(args.sizes, args.layers, room(64, 2048 + 256 + 16), 65)
        lens, pf, dec, kv = rig.unequal(64, 16, 2048, 256)
        tf = rig.prefill_flops(lens) / (pf / 1e3) / 1e12
        gbs = (rig.model.weight_bytes() + kv) / (dec / 1e3) / 1e9
        print(json.dumps({"only": "unequal", "sizes": args.sizes, "prompts": 64, "tokens": sum(lens),
                          "layers": rig.layers, "prefill_ms": pf, "prefill_tok_s": sum(lens) / (pf / 1e3),
                          "prefill_tflops": tf, "prefill_frac": tf / bf16_tf, "decode_ms_per_step": dec,
                          "decode_tok_s": 64 / (dec / 1e3), "decode_gb_s": gbs, "decode_hbm_frac": gbs / hbm_gbs}))
        return 0

    # ---- the headline: decode at the default batch and context -----------------------------------------------------
    big = B if args.no_points else max(B, 64)
    rig = Rig(HEADLINE, args.layers, room(big, C), big + 1)
    cfg, engine, model, E = rig.cfg, rig.engine, rig.model, rig.E
    clocks = ClockSampler()
    clocks.start()
    ms, launches, kv_bytes = rig.decode(B, C, Kst, W)
    clk = clocks.stop()
    ms_step = ms / Kst
    value = B * Kst / (ms / 1e3)
    step_bytes = model.weight_bytes() + kv_bytes
    achieved = step_bytes / (ms_step / 1e3) / 1e9

    # ---- end to end through Engine.generate --------------------------------------------------------------------
    n_new = Kst + W
    e2e_prompts = rig.prompts(B, C - n_new)
    e2e_opt = E.GenerateOptions(max_tokens=n_new, ignore_eos=True, max_batch=B)
    from exl3_server_b200.engine.decode import TRANSFERRED

    def timed_generate(opt):
        before = dict(TRANSFERRED)
        res = engine.generate(e2e_prompts, opt)
        steps = max(r.completion_tokens for r in res) - 1
        rate = sum(r.completion_tokens - 1 for r in res) / max(r.decode_seconds for r in res)
        return rate, (TRANSFERRED["h2d"] - before["h2d"]) / steps, (TRANSFERRED["d2h"] - before["d2h"]) / steps

    engine.generate(e2e_prompts, e2e_opt)               # untimed: records the decode graph this shape needs
    # default user path: greedy, the next step is launched before the host reads the last one's ids
    e2e, h2d, d2h = timed_generate(e2e_opt)
    # the same with the host feeding every step's token ids (what sampling with filters does)
    fed_opt = E.GenerateOptions(max_tokens=n_new, ignore_eos=True, max_batch=B, run_ahead=False)
    e2e_fed, h2d_fed, d2h_fed = timed_generate(fed_opt)

    # ---- prefill of one prompt ---------------------------------------------------------------------------------------
    T = args.prefill_tokens
    pf_ms = rig.prefill(T)
    flops = rig.prefill_flops([T])
    prefill_rec = {"value": T / (pf_ms / 1e3), "tokens": T, "ms": pf_ms,
                   "frac": flops / (pf_ms / 1e3) / (bf16_tf * 1e12), "tflops": flops / (pf_ms / 1e3) / 1e12}

    points, fracs = {}, {}

    def point(name, got):
        points[name], fracs[name] = got

    if not args.no_points:
        st = max(8, Kst // 2)
        point("decode_b1", rig.decode_point("2B b1 ctx %d" % C, 1, C, st, 3, hbm_gbs))
        point("decode_b64", rig.decode_point("2B b64 ctx %d" % C, 64, C, st, 3, hbm_gbs))
        # the other contexts the baseline's table names
        for b, c in ((1, 128), (8, 128), (1, 2048), (8, 2048), (64, 2048)):
            point(f"decode_b{b}_ctx{c}", rig.decode_point(f"2B b{b} ctx {c}", b, c, min(st, c - 16), 3, hbm_gbs))
        # longer contexts: a prompt of 8,192 tokens, and decoding at 16,384 tokens (the cache is then 0.9 of the bytes)
        if big * C >= 8 * 16384 + 8192:
            point("decode_b8_ctx16384", rig.decode_point("2B b8 ctx 16384", 8, 16384, 16, 3, hbm_gbs, repeats=1))
            ms_long = rig.prefill(8192, repeats=2, warm=1)
            point("prefill_8192", (8192 / (ms_long / 1e3),
                                   rig.prefill_flops([8192]) / (ms_long / 1e3) / 1e12 / bf16_tf))
    layers_run, layers_full = rig.layers, rig.layers_full
    del engine, model
    rig.close()

    if not args.no_points:
        # ---- MiniCPM4-8B sizes: 16 query heads per key/value head of 128, untied head ---------------------------
        r8 = Rig("minicpm4-8b", 0, room(64, 2048), 65)
        for b in (1, 8, 64):
            point(f"m4_8b_decode_b{b}_ctx2048", r8.decode_point(f"8B b{b} ctx 2048", b, 2048, 24, 3, hbm_gbs))
        point("m4_8b_decode_b1_ctx128", r8.decode_point("8B b1 ctx 128", 1, 128, 24, 3, hbm_gbs))
        ms8 = r8.prefill(2048)
        tf8 = r8.prefill_flops([2048]) / (ms8 / 1e3) / 1e12
        point("m4_8b_prefill_2048", (2048 / (ms8 / 1e3), tf8 / bf16_tf))
        r8.close()
        # ---- MiniCPM4-0.5B sizes: 64 prompts of 16 to 2,048 tokens in one step, then 256 decode steps ------------
        r05 = Rig("minicpm4-0.5b", 0, room(64, 2048 + 256 + 16), 65)
        lens, pf, dec, kv = r05.unequal(64, 16, 2048, 256)
        point("m4_05b_unequal64_prefill", (sum(lens) / (pf / 1e3),
                                           r05.prefill_flops(lens) / (pf / 1e3) / 1e12 / bf16_tf))
        point("m4_05b_unequal64_decode", (64 / (dec / 1e3),
                                          (r05.model.weight_bytes() + kv) / (dec / 1e3) / 1e9 / hbm_gbs))
        r05.close()

    out = {
        "metric": "decode tok/s (batch 8, context 4096, 2B-class MiniCPM, bf16)", "value": value, "unit": "tok/s",
        "n_gpus": 1, "steps": Kst, "warmup": W, "ms_per_step": ms_step, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights N(0,0.02), uniform random token ids, contexts prefilled by the engine",
        "config": {"model": "MiniCPM-2B layer sizes", "global_batch": B, "seq_len": C, "parallelism": "none",
                   "layers": layers_run, "layers_full": layers_full, "hidden": cfg.hidden_size,
                   "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "tied_head": True,
                   "rope_theta": cfg.rope_theta, "rms_norm_eps": cfg.rms_norm_eps, "page_size": page,
                   "l2": "inputs exceed L2 (weights and cache read per step)", "peaks": peak_src},
        "clocks": clk,
        "e2e": {"value": e2e, "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h,
                "host_fed": {"value": e2e_fed, "h2d_bytes_per_step": h2d_fed, "d2h_bytes_per_step": d2h_fed},
                "note": "decode tok/s inside Engine.generate after its prefill (prompts: host lists, one pinned "
                        "H2D copy); greedy ids feed the next step on the GPU and are read by the host every step"},
        "gpu_launches": int(launches),
        "prefill": prefill_rec,
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": hbm_gbs, "unit": "GB/s",
                     "frac": achieved / hbm_gbs, "bytes_per_step": step_bytes},
        "points": points,
        "points_frac": fracs,
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
