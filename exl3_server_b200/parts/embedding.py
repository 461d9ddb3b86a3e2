"""Token embedding and output head.

Embedding: ``h0[t] = E[id_t] * scale`` (the gather is src/model.cpp:529; the
scale is MiniCPM's ``scale_emb``).  Head: ``logits = (norm(h) / divisor) W^T``
in float32, computed only for the rows that were asked for (the reference
computes every row, src/model.cpp:589-592); ``W`` is the embedding table when
the head is tied.  With ``softcap`` c > 0 in the head's parameters the logits become ``c tanh(logits / c)``.

Both are registered part kinds like the others (``"table"`` and ``"linear"``).  An embedding of another kind has
``tensor_specs(spec)``, ``__init__(spec, tensors, ctx)`` and ``forward(token_ids) -> ResidualStream``; a head has
``tensor_specs(spec)``, ``__init__(spec, tensors, embedding, ctx)``, ``forward(stream, final_norm, rows) ->
float32 logits [rows, vocab]`` and ``read_bytes()``, the weight bytes a step reads.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..ops import kernels as K
from ..weights.loader import TensorSpec
from .base import BuildContext, ResidualStream, StateRequest
from .linear import Linear
from .norm import RMSNorm
from .registry import register_embedding, register_head
from .spec import EmbeddingSpec, HeadSpec


class Embedding:
    @staticmethod
    def tensor_specs(spec: EmbeddingSpec) -> List[TensorSpec]:
        return [TensorSpec(spec.name, (spec.vocab, spec.width))]

    def __init__(self, spec: EmbeddingSpec, tensors: Dict[str, torch.Tensor], ctx: BuildContext):
        self.spec = spec
        self.table = tensors[spec.name].to(ctx.dtype).contiguous()

    def forward(self, token_ids: torch.Tensor) -> ResidualStream:
        return ResidualStream(K.embed(token_ids, self.table, float(self.spec.scale)))

    def row_source(self):
        """``(table, scale)``: a token's embedding is its row of the table times the scale."""
        return self.table, float(self.spec.scale)

    def weight_bytes(self) -> int:
        return self.table.numel() * self.table.element_size()


class Head:
    @staticmethod
    def tensor_specs(spec: HeadSpec) -> List[TensorSpec]:
        if spec.tied:
            return []
        # tied None: the configuration does not say; a head of its own is used when the checkpoint has one
        return [TensorSpec(spec.name, (spec.vocab, spec.width), optional=spec.tied is None)]

    def __init__(self, spec: HeadSpec, tensors: Dict[str, torch.Tensor], embedding: Embedding, ctx: BuildContext):
        self.spec = spec
        self.tied = spec.tied if spec.tied is not None else spec.name not in tensors
        weight = embedding.table if self.tied else tensors[spec.name]
        self.linear = Linear(weight, None, ctx.dtype)
        if self.tied:
            self.linear.weight = embedding.table          # one copy in memory

    def forward(self, stream: ResidualStream, final_norm, rows: Optional[torch.Tensor]) -> torch.Tensor:
        r = final_norm.add_norm(stream, rows=rows, out_scale=1.0 / float(self.spec.input_divisor))
        logits = self.linear(r, out_dtype=torch.float32)
        cap = float(self.spec.params.get("softcap", 0.0))
        if cap > 0.0:
            K.softcap(logits, cap)              # logits <- cap * tanh(logits / cap)
        return logits

    def weight_bytes(self) -> int:
        """Bytes this part holds beyond the embedding's."""
        return 0 if self.tied else self.linear.weight_bytes()

    def read_bytes(self) -> int:
        """Weight bytes a step reads for the logits (a tied head reads the embedding table)."""
        return self.linear.weight_bytes()


class HashedPairEmbedding:
    """``h0[t] = E[id_t] + P[(id_(t-1) * mul_prev + id_t * mul_cur) mod buckets]``: the token's row plus a row of a
    second table picked by a hash of the token and the one before it; a sequence's first token takes the second
    table's last row (number ``buckets``).  The token before a step's first token is per-sequence state (an int32
    per slot) that the kernel keeps up.  Parameters of the spec: ``pair_name``, ``buckets``, ``mul_prev``,
    ``mul_cur``."""

    takes_batch = True

    @staticmethod
    def tensor_specs(spec: EmbeddingSpec) -> List[TensorSpec]:
        return [TensorSpec(spec.name, (spec.vocab, spec.width)),
                TensorSpec(spec.params["pair_name"], (int(spec.params["buckets"]) + 1, spec.width))]

    def __init__(self, spec: EmbeddingSpec, tensors: Dict[str, torch.Tensor], ctx: BuildContext):
        if float(spec.scale) != 1.0:
            raise ValueError("hashed pair embedding: no scale on the sum of two rows")
        self.spec = spec
        self.table = tensors[spec.name].to(ctx.dtype).contiguous()
        self.pairs = tensors[spec.params["pair_name"]].to(ctx.dtype).contiguous()
        self.buckets = int(spec.params["buckets"])
        self.mul_prev, self.mul_cur = int(spec.params["mul_prev"]), int(spec.params["mul_cur"])

    def state_request(self) -> StateRequest:
        return StateRequest((), torch.int32)

    def forward(self, token_ids: torch.Tensor, batch, state: Optional[torch.Tensor]) -> ResidualStream:
        if state is None:
            raise RuntimeError("the hashed pair embedding needs its per-sequence state")
        return ResidualStream(K.embed_hashed(token_ids, batch.tok_pos, batch.tok_seq, batch.row_start, batch.slot_ids,
                                             self.table, self.pairs, self.buckets, self.mul_prev, self.mul_cur, state))

    def weight_bytes(self) -> int:
        return (self.table.numel() + self.pairs.numel()) * self.table.element_size()


class SinusoidEmbedding:
    """``h0[t] = norm(E[id_t] * scale + P[p_t])``: the token's row plus a sinusoidal vector of its position, entry 2i
    ``sin(p base^(-2i / width))`` and entry 2i + 1 the cosine, then an RMS norm where the spec has one.  One kernel, float32
    inside; in the bfloat16 path it also leaves the row in 16 bits for the first layer.  Parameters of the spec: ``base``,
    ``norm`` (a ``NormSpec`` of kind ``rms``, or None) and ``norm_name``."""

    takes_batch = True

    @staticmethod
    def tensor_specs(spec: EmbeddingSpec) -> List[TensorSpec]:
        out = [TensorSpec(spec.name, (spec.vocab, spec.width))]
        if spec.params.get("norm") is not None:
            out += RMSNorm.tensor_specs(spec.params["norm"], spec.params["norm_name"])
        return out

    def __init__(self, spec: EmbeddingSpec, tensors: Dict[str, torch.Tensor], ctx: BuildContext):
        self.spec, self.dtype = spec, ctx.dtype
        self.table = tensors[spec.name].to(ctx.dtype).contiguous()
        i = torch.arange((spec.width + 1) // 2, dtype=torch.float64)
        base = torch.tensor(float(spec.params.get("base", 10000.0)), dtype=torch.float64)
        self.frequencies = K.rotary_table(torch.pow(base, -2.0 * i / spec.width)).to(ctx.device)
        self.norm_w, self.eps = None, 0.0
        norm = spec.params.get("norm")
        if norm is not None:
            if norm.kind != "rms":
                raise ValueError(f"sinusoid embedding: the norm must be of kind 'rms', got {norm.kind!r}")
            self.norm_w = RMSNorm(norm, tensors, spec.params["norm_name"], ctx).weight.float().contiguous()
            self.eps = norm.eps

    def forward(self, token_ids: torch.Tensor, batch, state: Optional[torch.Tensor]) -> ResidualStream:
        h, x = K.embed_sinusoid(token_ids, batch.tok_pos, self.table, float(self.spec.scale), self.frequencies, self.norm_w,
                                self.eps, self.dtype)
        stream = ResidualStream(h)
        stream.act = x if x is not None else h
        return stream

    def weight_bytes(self) -> int:
        return self.table.numel() * self.table.element_size()


register_embedding("table", Embedding)
register_embedding("table_sinusoid", SinusoidEmbedding)
register_embedding("table_hashed_pair", HashedPairEmbedding)
register_head("linear", Head)
