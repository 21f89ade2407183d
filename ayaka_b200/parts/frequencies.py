"""Rotary frequencies for contexts longer than the one they were chosen for."""

from __future__ import annotations

import math

__all__ = ["blended_frequencies"]


def blended_frequencies(dims: int, base: float, *, factor: float = 1.0, original: float = 0.0,
                        fast: float = 0.0, slow: float = 0.0) -> tuple[list[float], float]:
    """Rotary frequencies ``f_i = base^(-2i / dims)`` for the ``dims / 2`` pairs and the gain on
    cosine and sine. With ``factor`` > 1 the frequencies are blended for contexts longer than
    ``original``: a pair that makes ``t`` turns over ``original`` positions has the index
    ``d(t) = dims * ln(original / (2 pi t)) / (2 ln base)``; with ``lo = max(floor(d(fast)), 0)``,
    ``hi = min(ceil(d(slow)), dims - 1)`` and ``ramp_i = clamp((i - lo) / max(hi - lo, 0.001),
    0, 1)`` the frequency is ``f_i / factor * ramp_i + f_i * (1 - ramp_i)``, and the gain is
    ``0.1 * ln(factor) + 1``."""
    half = dims // 2
    freq = [float(base) ** (-2.0 * i / dims) for i in range(half)]
    if not factor or factor == 1.0 or not original:
        return freq, 1.0

    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0
