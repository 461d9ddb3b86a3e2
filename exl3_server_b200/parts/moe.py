"""A routed feed-forward (mixture of experts) with optional identity experts and a shared expert.

The router has ``experts + identity`` outputs: ``z = Wr r`` in float32, scores ``s = softmax(z)`` over all of them.
The choice is made by ``c = s + correction`` (a stored vector); the outputs form ``groups`` equal groups of
neighbours, a group's score is its largest ``c``, and only outputs of the ``keep`` best groups can be chosen (the
others count as minus infinity); the ``top`` largest ``c`` among them are the token's picks.  A pick's weight is its
score ``s`` (without the correction) times ``scale``; weights are not renormalised.  Picks below ``experts`` are
small feed-forwards ``Wd_e act(Wu_e r)`` without biases (tensors ``e<i>.up``, ``e<i>.down``); the last ``identity``
outputs have no tensors and stand for the input ``r`` itself.  The output is the weighted sum of the picks, plus, when
the spec has ``shared_inner``, a shared expert of the same form (``shared.up``, ``shared.down``) that every token
runs, times ``sigmoid(w_sg . r)`` (``shared.sg``, one number per token).

Variants: with ``score`` ``"picked"`` the choice is made by the logits themselves and a pick's weight is the softmax over
the chosen logits alone, times ``scale``; ``router_bias`` (with ``"picked"`` only) adds a stored bias ``router.b`` to the
logits.  ``correction`` False: there is no correction.  ``shared_gate`` False: the shared expert is added as it is.

Parameters of the spec: ``experts``, ``identity``, ``top``, ``scale``, ``groups``, ``keep``, ``activation`` (``gelu``,
``gelu_tanh``, ``silu`` or ``relu2``), ``score`` (``softmax``, ``sigmoid`` or ``picked``), ``group_score`` (``max``, or ``top2``: a group's
score is the sum of its two largest choice scores), ``shared_inner`` (0: none); ``inner`` is an expert's hidden size.
``expert`` = ``"clamped_glu"`` makes the experts (and the shared one) gated with a bounded gate, ``Wd (g sigmoid(alpha
g) (u + 1))``, ``g = min(Wg r, limit)``, ``u = clamp(Wu r, -limit, limit)`` (tensors ``e<i>.gate``, ``e<i>.up``,
``e<i>.down``; parameters ``limit``, ``shared_limit``, ``alpha``): gate and up are one stacked matrix per expert, the
activation a kernel of its own between the two grouped products.  ``expert`` = ``"glu"``: gated experts ``Wd (act(Wg r) *
(Wu r))`` (the same tensor names); gate and up rows alternate in one stacked matrix, so that the activation is the first
product's epilogue in all three of its kernels.  Tensors: ``router [experts + identity, width]``, ``correction [experts + identity]`` and the
experts'.

``table_routed``: there is no router.  An integer table ``table [vocab, top]`` gives every token id its ``top`` experts, each
with the weight ``1 / top`` (parameters ``vocab``, ``experts``, ``top``, ``expert``, ``activation``).  The plans of all such
layers of a model depend on the token ids alone: the first one that runs in a step has one kernel make them all
(``kernels.moe_table_plans``), for every pass over a layer that runs several times too.

How it runs (``csrc/moe.cu``): the router kernel also computes the shared expert's gate (its vector is one more row
of the router's float32 matrix); a one-block kernel orders the step's (token, pick) pairs by expert into tiles, on the
device, so a step is the same list of launches whatever the router chose (it can be part of a recorded graph); the
experts' weights are stacked ``[experts, out, in]`` and both projections are grouped products over the tiles; the
last kernel sums picks, identity picks and the gated shared expert in float32 (an arrangement that norms this part's output
asks for the pieces, ``forward_pieces``, and gets sum, norm and residual step from one kernel).  Which product runs depends on the
step only through its number of pairs: in bfloat16, few pairs (decode) take the kernel that reads each expert's
matrix once with a warp per output feature, many pairs (prompts) are gathered into the plan's order and go through
the tcgen05 grouped product; float32, and sizes those two do not take, use the CUDA-core tiles.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..ops import kernels as K
from ..weights.loader import TensorSpec
from .base import BuildContext
from .ffn import ClampedGLU, DenseFeedForward
from .registry import register_feed_forward
from .spec import FeedForwardSpec


FEW_PAIRS = 128       # up to here the few-row product; from MANY_PAIRS on the tensor cores
MANY_PAIRS = 512


class PickedSum:
    """``sum_k wt[t, k] y[t, k] + gate[t] shared[t]``, not summed yet."""

    def __init__(self, y, idx, wt, shared, gate, n_experts: int):
        self.y, self.idx, self.wt, self.shared, self.gate, self.n_experts = y, idx, wt, shared, gate, n_experts

    def norm_add(self, h: torch.Tensor, weight: torch.Tensor, eps: float, want_x: bool):
        return K.moe_combine_norm(self.y, self.idx, self.wt, self.shared, self.gate, self.n_experts, h, weight, eps, want_x)


class RoutedFeedForward:
    @staticmethod
    def _sizes(spec: FeedForwardSpec):
        p = spec.params
        return int(p["experts"]), int(p.get("identity", 0)), int(p.get("shared_inner", 0))

    @staticmethod
    def _clamped(spec: FeedForwardSpec) -> bool:
        return spec.params.get("expert", "dense") == "clamped_glu"

    @staticmethod
    def _glu(spec: FeedForwardSpec) -> bool:
        return spec.params.get("expert", "dense") == "glu"

    @classmethod
    def _expert_specs(cls, spec: FeedForwardSpec, prefix: str, n: int) -> List[TensorSpec]:
        out = []
        for e in range(n):
            if cls._clamped(spec) or cls._glu(spec):
                out.append(TensorSpec(f"{prefix}e{e}.gate", (spec.inner, spec.width)))
            out += [TensorSpec(f"{prefix}e{e}.up", (spec.inner, spec.width)),
                    TensorSpec(f"{prefix}e{e}.down", (spec.width, spec.inner))]
        return out

    @classmethod
    def _shared_spec(cls, spec: FeedForwardSpec, inner: int) -> FeedForwardSpec:
        if cls._clamped(spec):
            return FeedForwardSpec(kind="clamped_glu", width=spec.width, inner=inner,
                                   params={"limit": spec.params.get("shared_limit", spec.params["limit"]),
                                           "alpha": spec.params.get("alpha", ClampedGLU.ALPHA)})
        return FeedForwardSpec(kind="dense", width=spec.width, inner=inner,
                               params={"activation": spec.params.get("activation", "gelu")})

    @classmethod
    def _shared_class(cls, spec: FeedForwardSpec):
        return ClampedGLU if cls._clamped(spec) else DenseFeedForward

    @classmethod
    def tensor_specs(cls, spec: FeedForwardSpec, prefix: str) -> List[TensorSpec]:
        E, I, shared = cls._sizes(spec)
        out = [TensorSpec(prefix + "router", (E + I, spec.width))]
        if spec.params.get("correction", True):
            out.append(TensorSpec(prefix + "correction", (E + I,)))
        if spec.params.get("router_bias", False):
            out.append(TensorSpec(prefix + "router.b", (E + I,)))
        out += cls._expert_specs(spec, prefix, E)
        if shared:
            out += cls._shared_class(spec).tensor_specs(cls._shared_spec(spec, shared), prefix + "shared.")
            if spec.params.get("shared_gate", True):
                out.append(TensorSpec(prefix + "shared.sg", (1, spec.width)))
        return out

    def __init__(self, spec: FeedForwardSpec, tensors: Dict[str, torch.Tensor], prefix: str, ctx: BuildContext):
        E, I, shared = self._sizes(spec)
        p = spec.params
        self.spec, self.dtype = spec, ctx.dtype
        self.E, self.I = E, I
        self.top, self.scale = int(p["top"]), float(p.get("scale", 1.0))
        self.groups, self.keep = int(p.get("groups", 1)), int(p.get("keep", 1))
        self.act, self.score = p.get("activation", "gelu"), p.get("score", "softmax")
        self.group_score = p.get("group_score", "max")
        self._expert_form(spec)
        if self.glu and shared:
            raise ValueError("routed feed-forward: no shared expert beside experts of the form 'glu'")
        if self.act not in K.MOE_ACTIVATIONS or self.score not in K.MOE_SCORES or self.group_score not in K.MOE_GROUP_SCORES:
            raise ValueError(f"routed feed-forward: unknown activation {self.act!r}, score {self.score!r} or group "
                             f"score {self.group_score!r}")
        n = E + I
        if n < 1 or n % self.groups != 0 or not 1 <= self.keep <= self.groups or \
                not 1 <= self.top <= self.keep * (n // self.groups):
            raise ValueError(f"routed feed-forward: {n} outputs, {self.groups} groups, keep {self.keep}, top {self.top}")
        rows = [tensors[prefix + "router"].float()]
        self.shared = None
        if shared:
            self.shared = self._shared_class(spec)(self._shared_spec(spec, shared), tensors, prefix + "shared.", ctx)
            if p.get("shared_gate", True):
                rows.append(tensors[prefix + "shared.sg"].float().reshape(1, spec.width))
        self.gates = len(rows) - 1                                    # the shared expert's gate: one more router row
        self.router = torch.cat(rows, dim=0).contiguous()             # float32: the router is computed in 32 bits
        if p.get("router_bias", False) and (self.score != "picked" or p.get("correction", True)):
            raise ValueError("routed feed-forward: a bias of the logits goes with the score 'picked' and no correction")
        if p.get("correction", True):
            self.correction = tensors[prefix + "correction"].float().contiguous()
        elif p.get("router_bias", False):
            self.correction = tensors[prefix + "router.b"].float().contiguous()
        else:
            self.correction = torch.zeros(n, dtype=torch.float32, device=self.router.device)
        self.w_up = self.w_down = None
        if E:
            self._stack_experts(tensors, prefix, E, ctx)

    def _expert_form(self, spec: FeedForwardSpec) -> None:
        p = spec.params
        self.clamped, self.glu = self._clamped(spec), self._glu(spec)
        if self.clamped:
            self.act = "none"                  # the bounded gate is applied between the two products
            self.limit, self.alpha = float(p["limit"]), float(p.get("alpha", ClampedGLU.ALPHA))

    def _stack_experts(self, tensors: Dict[str, torch.Tensor], prefix: str, E: int, ctx: BuildContext) -> None:
        get = lambda e, name: tensors[f"{prefix}e{e}.{name}"].to(ctx.dtype)
        if self.clamped:                       # [gate; up] rows of every expert
            ups = [torch.cat([get(e, "gate"), get(e, "up")], dim=0) for e in range(E)]
        elif self.glu:                         # gate and up rows in turn
            ups = [torch.stack([get(e, "gate"), get(e, "up")], dim=1).reshape(-1, self.spec.width) for e in range(E)]
        else:
            ups = [get(e, "up") for e in range(E)]
        self.w_up = torch.stack(ups).contiguous()
        self.w_down = torch.stack([get(e, "down") for e in range(E)]).contiguous()

    def _pieces(self, x: torch.Tensor, batch):
        idx, wt, gate = K.moe_route(x, self.router, self.correction, self.E + self.I, self.gates,
                                    self.groups, self.keep, self.top, self.scale, self.score, self.group_score)
        y = None
        if self.E:
            y = self._experts(x, idx.numel(), lambda kind: K.moe_plan(idx, self.E, K.moe_tile_rows(kind)))
        s = self.shared.forward(x, batch) if self.shared is not None else None
        return y, idx, wt, s, gate

    def forward(self, x: torch.Tensor, batch) -> torch.Tensor:
        y, idx, wt, s, gate = self._pieces(x, batch)
        return K.moe_combine(y, idx, wt, x, s, gate, self.E)

    def forward_pieces(self, x: torch.Tensor, batch):
        """The output as the pieces of its weighted sum, for a caller whose next step takes them (see
        ``RMSNorm.add_normed``); the output itself where there are identity experts or odd sizes."""
        if self.I or not self.E or not K.moe_combine_norm_supported(x.shape[1]):
            return self.forward(x, batch)
        return PickedSum(*self._pieces(x, batch), n_experts=self.E)

    def _product(self, pairs: int) -> str:
        """Which of the experts' products (``kernels.moe_tile_rows``) takes a step of so many pairs."""
        width, inner = self.w_up.shape[2], self.w_down.shape[2]
        if self.dtype == torch.bfloat16 and width % 8 == 0 and inner % 8 == 0:
            if pairs >= MANY_PAIRS and K.moe_tc_supported(self.dtype, inner, width):
                return "tc"
            if pairs <= FEW_PAIRS:
                return "few"
        return "tile"

    def _experts(self, x: torch.Tensor, pairs: int, plan_for) -> torch.Tensor:
        """float32 ``[pairs, width]``: every planned pair's expert output at the pair's own place.  ``plan_for(kind)``: the
        step's ``(order, plan)`` with the tiles of that product."""
        gated = (lambda mid: K.clamped_glu(mid, self.limit, self.alpha, self.dtype)) if self.clamped else (lambda mid: mid)
        kind = self._product(pairs)
        if kind != "tile" and (x.dtype != torch.bfloat16 or x.stride(0) % 8 != 0):
            x = x.to(torch.bfloat16).contiguous()
        order, plan = plan_for(kind)
        if kind == "tc":
            xs = K.moe_gather(x, self.top, order, plan)
            mid = gated(K.moe_gemm_tc(xs, self.w_up, order, plan, self.dtype, act=self.act, glu=self.glu))
            return K.moe_gemm_tc(mid, self.w_down, order, plan, torch.float32)
        product = K.moe_gemv if kind == "few" else K.moe_gemm
        mid = gated(product(x, self.top, self.w_up, order, plan, self.dtype, act=self.act, glu=self.glu))
        return product(mid, 1, self.w_down, order, plan, torch.float32)

    def untouched_bytes(self, tokens: int) -> int:
        """Bytes of experts' matrices that a step of ``tokens`` tokens is not expected to read when every router output
        is as likely a pick as any other (random weights): an output stays unpicked by a token with probability
        ``1 - top / outputs``."""
        if self.w_up is None:
            return 0
        per_expert = (self.w_up[0].numel() + self.w_down[0].numel()) * self.w_up.element_size()
        return int(self.E * per_expert * (1.0 - self.top / (self.E + self.I)) ** tokens)

    def weight_bytes(self) -> int:
        """Weight bytes a token's step reads at most: the router, the shared expert and ``top`` experts per token
        (a step of many tokens reads each expert once; this counts the matrices once)."""
        n = self.router.numel() * 4 + self.correction.numel() * 4
        if self.w_up is not None:
            n += (self.w_up.numel() + self.w_down.numel()) * self.w_up.element_size()
        if self.shared is not None:
            n += self.shared.weight_bytes()
        return n


class TableRoutedFeedForward(RoutedFeedForward):
    @classmethod
    def tensor_specs(cls, spec: FeedForwardSpec, prefix: str) -> List[TensorSpec]:
        E, top = int(spec.params["experts"]), int(spec.params["top"])
        return cls._expert_specs(spec, prefix, E) + \
            [TensorSpec(prefix + "table", (int(spec.params["vocab"]), top), kind="int", high=E)]

    def __init__(self, spec: FeedForwardSpec, tensors: Dict[str, torch.Tensor], prefix: str, ctx: BuildContext):
        p = spec.params
        self.spec, self.dtype = spec, ctx.dtype
        self.E, self.I, self.top = int(p["experts"]), 0, int(p["top"])
        self.act = p.get("activation", "silu")
        self._expert_form(spec)
        if self.act not in K.MOE_ACTIVATIONS or not 1 <= self.top <= self.E:
            raise ValueError(f"table-routed feed-forward: activation {self.act!r}, {self.E} experts, top {self.top}")
        self.shared = None
        self.table = tensors[prefix + "table"].to(torch.int32).contiguous()
        if self.table.numel() and not (0 <= int(self.table.min()) and int(self.table.max()) < self.E):
            raise ValueError(f"{prefix}table: entries must lie below the {self.E} experts")
        self._stack_experts(tensors, prefix, self.E, ctx)
        # all layers of this kind in the model: their plans are made together
        self.peers = ctx.shared.setdefault("table_routed", [])
        self.place = len(self.peers)
        self.peers.append((self.table, self.E, self.top, self._product))

    def _plan(self, batch):
        plans = batch.memo.get("table_routed")
        if plans is None:
            T = batch.token_ids.numel()
            plans = batch.memo["table_routed"] = K.moe_table_plans(
                batch.token_ids, [(table, E, K.moe_tile_rows(product(T * top))) for table, E, top, product in self.peers])
        return plans[self.place]

    def forward_picks(self, x: torch.Tensor, batch):
        """``(y float32 [T * top, width], top, weight)``: the output is ``weight * sum_k y[t * top + k]``, which the caller's
        next kernel adds up."""
        return self._experts(x, x.shape[0] * self.top, lambda kind: self._plan(batch)), self.top, 1.0 / self.top

    def forward(self, x: torch.Tensor, batch) -> torch.Tensor:
        out = torch.zeros((x.shape[0], self.spec.width), dtype=torch.float32, device=x.device)
        K.residual_step(out, picks=self.forward_picks(x, batch))
        return out

    def weight_bytes(self) -> int:
        return (self.w_up.numel() + self.w_down.numel()) * self.w_up.element_size()


register_feed_forward("routed", RoutedFeedForward)
register_feed_forward("table_routed", TableRoutedFeedForward)
