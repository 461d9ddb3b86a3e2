"""A plain, slow implementation of the Soporax decoder: whole sequences, no cache, float64, one function per mechanism.
It shares no code with the package: config.json is read with ``json``, the weights with the ``safetensors`` library, and
everything is plain torch arithmetic on the CPU.  Attention builds the full score matrix head by head with its mask; the
latent attention forms every head's keys and values; experts run one by one on the tokens whose rows list them.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch
from safetensors import safe_open

F = torch.float64


def read_weights(model_dir: str) -> Dict[str, torch.Tensor]:
    out = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for k in f.keys():
            t = f.get_tensor(k)
            out[k] = t.to(F) if t.is_floating_point() else t.long()
    return out


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def base_frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequencies(dims: int, base: float, s: Optional[dict]) -> List[float]:
    """Frequencies whose wavelength is short are kept, long ones divided, and a straight line joins the two."""
    out = []
    for f in base_frequencies(dims, base):
        if s:
            wave = 2.0 * math.pi / f
            if wave < s["original"] / s["high"]:
                pass
            elif wave > s["original"] / s["low"]:
                f = f / s["factor"]
            else:
                part = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - part) * f / s["factor"] + part * f
        out.append(f)
    return out


def ramped_frequencies(dims: int, base: float, s: Optional[dict]):
    """(frequencies, factor on sines and cosines) with a ramp over the pairs' numbers (YaRN)."""
    freqs = base_frequencies(dims, base)
    if not s:
        return freqs, 1.0
    pair_of = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_neighbours(x: torch.Tensor, freqs: List[float], mult: float = 1.0) -> torch.Tensor:
    """x [T, ..., n]: features 2i and 2i + 1 of the first 2 len(freqs) turned by position times frequency i."""
    y = x.clone()
    at = torch.arange(x.shape[0], dtype=F).view(-1, *[1] * (x.dim() - 2))
    for i, f in enumerate(freqs):
        c, s = mult * torch.cos(at * f), mult * torch.sin(at * f)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def visible(T: int, window: int = 0) -> torch.Tensor:
    """[T, T]: whether query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i - j < window) if window else ok


def softmax_with_sink(s: torch.Tensor, ok: torch.Tensor, sink: Optional[float]) -> torch.Tensor:
    """Rows of s over the visible keys; ``sink``: the score of one more key that only takes weight, or None."""
    s = s.masked_fill(~ok, -math.inf)
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(torch.as_tensor(sink, dtype=F) - top)
    return e / den


def windowed_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """No positions, unit-length queries and keys, a window, a learned sink per head."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).view(T, H, d), eps)
    k = unit_rms((h @ w[p + "k"].T).view(T, G, d), eps)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    ok = visible(T, m["mask"]["size"] if m.get("mask") else 0)
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        outs.append(softmax_with_sink((q[:, hd] @ k[:, g].T) * m["scale"], ok, float(w[p + "sink"][hd])) @ v[:, g])
    return torch.cat(outs, dim=-1) @ w[p + "o"].T


def rotated_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Biases, banded rotary positions on part of a head, one added to the denominator, a gate per head."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freqs = banded_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling")) if m.get("rot") else []
    q = rotate_neighbours((h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d), freqs)
    k = rotate_neighbours((h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d), freqs)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    ok = visible(T)
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        o = softmax_with_sink((q[:, hd] @ k[:, g].T) * m["scale"], ok, 0.0) @ v[:, g]
        outs.append(o * gate[:, hd:hd + 1])
    return torch.cat(outs, dim=-1) @ w[p + "o"].T


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Queries, keys and values through latents, one rotated key part for all heads, a gate per output feature."""
    T, H, d, rd, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freqs, mult = ramped_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling")) if m.get("rot") else ([], 1.0)
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d + rd)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    k_rot = rotate_neighbours(down[:, r:], freqs, mult)
    q_rot = rotate_neighbours(q[:, :, d:], freqs, mult)
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    ok = visible(T)
    outs = []
    for hd in range(H):
        s = (q[:, hd, :d] @ k[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]
        outs.append(softmax_with_sink(s, ok, None) @ v[:, hd])
    return (torch.cat(outs, dim=-1) * gate) @ w[p + "o"].T


MIXERS = {"attention": windowed_attention, "attention_2": rotated_attention, "latent_attention": latent_attention}


def clamped_feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def expert(x: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    z = x @ w[p + "gate"].T
    return (z * torch.sigmoid(z) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def experts_by_table(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, tokens: List[int]) -> torch.Tensor:
    """The mean of the experts that the token's row of the table lists."""
    out = torch.zeros_like(h)
    rows = [w[p + "table"][tok].tolist() for tok in tokens]
    for e in sorted({e for picks in rows for e in picks}):
        at = [t for t, picks in enumerate(rows) if e in picks]
        out[at] += expert(h[at], w, f"{p}e{e}.") / len(rows[0])
    return out


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: Optional[dict], tokens: List[int]) -> torch.Tensor:
    if mlp is None:
        return torch.zeros_like(h)
    if mlp["kind"] == "dense":
        return clamped_feed_forward(h, w, p, mlp["limit"])
    return experts_by_table(h, w, p, tokens)


def layer_runs(cfg: dict) -> List[tuple]:
    """(layer, pass or None) in the order they run; a pass's number stands at its first layer only."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one whole sequence."""
    eps = cfg["norm"]["eps"]
    start = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = start
    for i, t in layer_runs(cfg):
        if t is not None:
            if t > 0:
                x = x + start
            x = x + w["loop.step"][t]
        layer = cfg["layers"][i]
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        x = x + (MIXERS[layer["type"]](h, w, f"l{i}.mix.", layer["mixer"], eps)
                 + feed_forward(h, w, f"l{i}.mlp.", layer.get("mlp"), tokens))
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg.get("logit_scale", 1.0)


class PlainSoporax:
    def __init__(self, model_dir: str):
        with open(os.path.join(model_dir, "config.json")) as f:
            self.cfg = json.load(f)
        self.w = read_weights(model_dir)
        self._memo: dict = {}

    def logits(self, tokens: List[int]) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._memo:
            self._memo[key] = forward(self.cfg, self.w, tokens)
        return self._memo[key]

    def layers(self, tokens: List[int]) -> torch.Tensor:
        out: list = []
        forward(self.cfg, self.w, tokens, out)
        return torch.stack(out)

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(torch.argmax(forward(self.cfg, self.w, toks)[-1])))
        return toks[len(prompt):]
