"""Rows of a learned table by the distance between a query and a key.

A table of ``rows`` rows with a largest distance ``far`` serves, with h = rows // 2: every distance n < h by a row of
its own, and from there on row h + floor(ln(n / h) / ln(far / h) * (rows - h)), at most the last one.  The borders are
found in whole numbers ((n / h)^m >= (far / h)^k with m = rows - h), so no rounding of a logarithm moves one.
"""
from __future__ import annotations

from fractions import Fraction
from typing import List

import torch


def bucket_starts(rows: int, far) -> List[int]:
    """The first distance of every row (rows that no distance reaches start where the next one does)."""
    half = rows // 2
    if rows < 1:
        raise ValueError(f"a table of distances needs rows, got {rows}")
    if half == 0:
        return [0] * rows
    far = Fraction(far)
    if far <= half:
        raise ValueError(f"a table of {rows} rows needs a largest distance above {half}, got {float(far)}")
    m = rows - half
    starts = list(range(half))
    for k in range(m):
        bound = far ** k * Fraction(half) ** (m - k)          # row half + k starts at the first n with n^m >= bound
        lo, hi = half - 1, int(far) + 1
        while hi - lo > 1:
            mid = (lo + hi) // 2
            if Fraction(mid) ** m >= bound:
                hi = mid
            else:
                lo = mid
        starts.append(hi)
    return starts


def spread_over_distances(table: torch.Tensor, far) -> torch.Tensor:
    """``table`` [rows, heads] as float32 [heads, n]: entry d of a head is its bias at distance d, the last entry serves
    every distance from n - 1 on."""
    rows = table.shape[0]
    starts = bucket_starts(rows, far)
    n = starts[-1] + 1
    which = torch.bucketize(torch.arange(n), torch.tensor(starts), right=True) - 1
    return table.float()[which.to(table.device)].t().contiguous()
