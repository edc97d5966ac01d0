"""Frequencies of rotary positions, as a mixer's configuration gives them.

Pair ``i`` of ``dims / 2`` turns by ``position * f_i`` with ``f_i = base ** (-2 i / dims)``.  With ``scaling`` (YaRN:
``factor``, ``original``, ``fast``, ``slow``) a pair that makes more than ``fast`` turns over ``original`` positions keeps
its frequency, one that makes fewer than ``slow`` turns is slowed by ``factor``, and a linear ramp over the pair's number
lies between; cosine and sine then come with the factor ``0.1 ln(factor) + 1``.
"""

from __future__ import annotations

import math
from typing import Mapping

SCALING_KEYS = ("factor", "original", "fast", "slow")


def rotary_frequencies(dims: int, base: float, scaling: Mapping[str, float] | None = None) -> tuple[list[float], float]:
    """``(f_0 .. f_(dims/2 - 1), factor on cosine and sine)``."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0
    factor, original, fast, slow = (float(scaling[k]) for k in SCALING_KEYS)

    def pair_with(turns: float) -> float:      # the (fractional) pair that makes so many turns over `original` positions
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(pair_with(fast)), 0)
    high = min(math.ceil(pair_with(slow)), dims - 1)
    span = max(high - low, 0.001)
    ramp = [min(max((i - low) / span, 0.0), 1.0) for i in range(dims // 2)]
    return [f / factor * r + f * (1.0 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(factor) + 1.0
