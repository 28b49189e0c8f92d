"""Learned biases of attention scores by the distance between query and key.

A table has one row of numbers (one a head) for each of ``rows`` buckets of distances: half of them one distance each
(0 .. rows/2 - 1), the others logarithmically wider up to the distance ``reach``; the last one takes every distance from there on:

    bucket(n) = n                                                        n < h = rows / 2
    bucket(n) = min(rows - 1, h + floor((rows - h) ln(n / h) / ln(reach / h)))   else

Buckets never fall as the distance grows, so the kernels get the numbers spread out by distance, up to the first distance of the
last bucket (``bias_table``), and need no logarithm.
"""

from __future__ import annotations

from typing import List

import torch

from ..ops import BIAS_BACK, BIAS_FRONT


def check_bucket_sizes(rows: int, reach: int) -> None:
    if rows < 2 or rows % 2:
        raise ValueError(f"a table of distance biases has an even number of rows, at least 2, got {rows}")
    if reach <= rows // 2:
        raise ValueError(f"distance biases that end at a distance of {reach} do not fit {rows} rows: half of the rows are one distance each")


def first_distances(rows: int, reach: int) -> List[int]:
    """The smallest distance that falls into bucket b or a later one, for every b: where floor((rows - h) ln(n / h) / ln(reach / h))
    comes to k, which is where (n / h)^(rows - h) comes to (reach / h)^k.  Whole numbers decide it, so no rounding moves a bucket."""
    check_bucket_sizes(rows, reach)
    h = rows // 2
    wide = rows - h
    out = list(range(h))
    for k in range(wide):
        need = reach ** k * h ** (wide - k)       # n^wide >= reach^k h^(wide - k)
        lo, hi = h, reach
        while lo < hi:
            mid = (lo + hi) // 2
            if mid ** wide >= need:
                hi = mid
            else:
                lo = mid + 1
        out.append(lo)
    return out


def bias_table(rel: torch.Tensor, reach: int, heads: int, kv_heads: int, factor: float = 1.0) -> torch.Tensor:
    """What the attention kernels take: [kv heads, BIAS_FRONT + distances + BIAS_BACK, heads a kv head] float32, the numbers of ``rel``
    [rows, heads] times ``factor``, the distance 0 at entry BIAS_FRONT; the entries ahead repeat it (positions past a row's own, which
    are masked), those behind repeat the last bucket's."""
    rows = rel.shape[0]
    firsts = first_distances(rows, reach)
    bucket: List[int] = []
    for b in range(rows):
        until = firsts[b + 1] if b + 1 < rows else firsts[b] + 1
        bucket += [b] * (until - firsts[b])
    index = [0] * BIAS_FRONT + bucket + [rows - 1] * BIAS_BACK
    spread = rel.float()[torch.tensor(index, dtype=torch.long, device=rel.device)] * float(factor)         # [entries, heads]
    return spread.reshape(len(index), kv_heads, heads // kv_heads).permute(1, 0, 2).contiguous()
