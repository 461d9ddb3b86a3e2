"""A learned bias of attention scores by distance.

A table ``rel [rows, heads]`` holds a number per bucket of distances and query head; ``rel[bucket(n), h]`` is added to the
score of the key n positions back.  With ``half = rows // 2`` and a largest distance D: the first ``half`` buckets hold one
distance each, ``bucket(n) = n``; the others' distances grow geometrically, ``bucket(n) = half + floor((rows - half)
ln(n / half) / ln(D / half))``, and everything from D on shares the last one.

The buckets' first distances are worked out once, in whole numbers, so that a distance that is exactly a power lands in its
own bucket whatever a logarithm rounds to.  Kernels get the biases by distance (``kernels.distance_table``), relative to the
last bucket's: ``near [heads, n]`` for the distances before the last bucket, ``far [heads]`` for all others.
"""
from __future__ import annotations

import math
from fractions import Fraction
from typing import List

import torch

from ..weights.loader import TensorSpec


def bucket_starts(rows: int, limit) -> List[int]:
    """The first distance of every bucket.  A bucket that no distance reaches starts where the next one does."""
    half = rows // 2
    if rows < 2:
        return [0] * rows
    top = Fraction(limit)
    if not top > half:
        raise ValueError(f"distance bias: the largest distance {limit} must lie beyond the table's first half, {half}")
    wide = rows - half
    ratio, base = top / half, Fraction(half)
    starts = list(range(half))
    for k in range(wide):
        # the smallest n >= half with (n / half)^wide >= ratio^k
        bound = ratio ** k * base ** wide
        n = max(half, math.floor(half * float(ratio) ** (k / wide)) - 2)
        while Fraction(n) ** wide < bound:
            n += 1
        starts.append(n)
    return starts


class DistanceBias:
    @staticmethod
    def tensor_spec(name: str, heads: int) -> TensorSpec:
        return TensorSpec(name, (-1, heads), free_dim=24)          # the table's length is the checkpoint's

    def __init__(self, rel: torch.Tensor, limit):
        rows, heads = rel.shape
        starts = bucket_starts(rows, limit)
        rel = rel.detach().double().cpu()
        n = starts[-1] if starts else 0                            # distances before the last bucket
        which = torch.zeros(n, dtype=torch.long)
        for b, s in enumerate(starts):
            which[s:] = b
        self.far = rel[-1].clone()
        self.near = (rel[which] - rel[-1]).T.contiguous() if n else torch.zeros(heads, 0, dtype=torch.float64)
