"""A plain, slow implementation of the Tunavik decoder: whole sequences, no cache, float64, one function per mechanism.
It shares no code with the package: config.json is read with ``json``, the weights with the ``safetensors`` library, and
everything is plain torch arithmetic on the CPU.  Attention builds the full score matrix with its mask and distance
biases; distances get their buckets one by one; the router is a loop over tokens.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Tuple

import torch
from safetensors import safe_open

F = torch.float64


def read_weights(model_dir: str) -> Dict[str, torch.Tensor]:
    out = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for k in f.keys():
            out[k] = f.get_tensor(k).to(F)
    return out


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def model_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight lies around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def sinusoids(T: int, width: int) -> torch.Tensor:
    """[T, width]: sines at even entries, cosines at odd ones, wavelengths from 2 pi up to 10000 times that."""
    out = torch.zeros(T, width, dtype=F)
    for i in range(width):
        a = torch.arange(T, dtype=F) * 10000.0 ** (-2.0 * (i // 2) / width)
        out[:, i] = torch.sin(a) if i % 2 == 0 else torch.cos(a)
    return out


def bucket(n: int, rows: int, limit: float) -> int:
    """The row of the distance table for a key n positions back: one row a distance for the first half of the table,
    then rows whose distances grow geometrically up to ``limit``, and the last row for everything beyond."""
    half = rows // 2
    if n < half:
        return n
    x = math.log(n / half) / math.log(limit / half) * (rows - half)
    if abs(x - round(x)) < 1e-9:                    # an exact power: not below its row through rounding
        x = round(x)
    return min(rows - 1, half + math.floor(x))


def temperature(T: int, coef: float, every: float) -> torch.Tensor:
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)], dtype=F)


def keys_and_values(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """[T, G, d] keys after their norm over all heads together, and [T, G, dv] values."""
    T = h.shape[0]
    k = unit_rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    return k.view(T, m["kv_heads"], m["dim"]), v.view(T, m["kv_heads"], m["vdim"])


def distance_bias(rel: torch.Tensor, T: int, limit: float) -> torch.Tensor:
    """[T, T, H]: rel[bucket(i - j)] for j <= i, zeros elsewhere."""
    rows = torch.tensor([bucket(n, rel.shape[0], limit) for n in range(T)])
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    d = (i - j).clamp(min=0)
    return rel[rows[d]]


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, kv,
              scores_out: Optional[list] = None) -> torch.Tensor:
    """``kv``: the keys and values to attend to (this layer's own or an earlier layer's)."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = unit_rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    if m.get("q_temp"):
        q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    q = q.view(T, H, d)
    k, v = kv
    bias = distance_bias(w[p + "rel"], T, m["bias_max"])
    hidden = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    outs = []
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * m["scale"] + bias[:, :, hd]
        if scores_out is not None:
            scores_out.append(s.clone())
        s = s.masked_fill(hidden, -math.inf)
        top = s.max(dim=-1, keepdim=True).values
        e = torch.exp(s - top)
        den = e.sum(dim=-1, keepdim=True) + torch.exp(w[p + "sink"][hd] - top)
        outs.append((e / den) @ v[:, g])
    return torch.cat(outs, dim=-1) @ w[p + "o"].T + w[p + "o.b"]


def relu2_expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def route(z: torch.Tensor, top: int) -> Tuple[List[int], torch.Tensor, float]:
    """One token's picks from its router logits, their weights, and the margin of the closest decision."""
    ranked = sorted(range(z.numel()), key=lambda e: (-float(z[e]), e))
    margin = float(z[ranked[top - 1]] - z[ranked[top]]) if top < len(ranked) else float("inf")
    picks = ranked[:top]
    return picks, torch.softmax(z[picks], dim=0), margin


def mixture_of_experts(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict,
                       margins: Optional[list] = None) -> torch.Tensor:
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = torch.zeros_like(h)
    chosen: Dict[int, list] = {}
    for t in range(h.shape[0]):
        picks, weights, margin = route(z[t], mlp["router"]["top"])
        if margins is not None:
            margins.append(margin)
        for e, c in zip(picks, weights):
            chosen.setdefault(e, []).append((t, c))
    for e, pairs in chosen.items():
        rows = torch.tensor([t for t, _ in pairs])
        y = relu2_expert(h[rows], w, f"{p}e{e}.")
        out.index_add_(0, rows, y * torch.stack([c for _, c in pairs])[:, None])
    if mlp.get("shared"):
        out = out + relu2_expert(h, w, p + "shared.")
    return out


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one whole sequence."""
    eps = cfg["norm"]["eps"]
    T = len(tokens)
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = model_norm(x + sinusoids(T, x.shape[1]), w["embed.norm"], eps)
    kept: dict = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        src = m.get("kv_from")
        if src is None:
            kept[i] = keys_and_values(x, w, p + "mix.", m, eps)
        y = attention(x, w, p + "mix.", m, eps, kept[i if src is None else src])
        x = x + model_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + model_norm(mixture_of_experts(x, w, p + "mlp.", layer["mlp"], margins), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    logits = model_norm(x, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


class PlainTunavik:
    def __init__(self, model_dir: str):
        with open(os.path.join(model_dir, "config.json")) as f:
            self.cfg = json.load(f)
        self.w = read_weights(model_dir)
        self._memo: dict = {}

    def run(self, tokens: List[int]) -> Tuple[torch.Tensor, float]:
        """(logits, the smallest margin of any router's decision over the sequence; infinite without routers)."""
        key = tuple(tokens)
        if key not in self._memo:
            margins: list = []
            self._memo[key] = (forward(self.cfg, self.w, tokens, None, margins), min(margins, default=float("inf")))
        return self._memo[key]

    def logits(self, tokens: List[int]) -> torch.Tensor:
        return self.run(tokens)[0]

    def closest_call(self, tokens: List[int]) -> float:
        return self.run(tokens)[1]

    def layers(self, tokens: List[int]) -> torch.Tensor:
        out: list = []
        forward(self.cfg, self.w, tokens, out)
        return torch.stack(out)

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(torch.argmax(forward(self.cfg, self.w, toks)[-1])))
        return toks[len(prompt):]
