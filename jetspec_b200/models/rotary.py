"""Rotary position tables: which entries of a head form a pair, how fast each pair turns, and frequency scalings.

A mixer names its rotation by a :class:`RotaryConfig`; :meth:`RotaryConfig.frequencies` and :meth:`RotaryConfig.amplitude`
are everything the ops and kernels need.  Tables are evaluated in double precision and rounded to fp32 once.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Union


@dataclass(frozen=True)
class BandScaling:
    """Pairs of wavelengths below ``original / high`` keep their frequency, those above ``original / low`` have it divided by
    ``factor``; between the two it is interpolated in ``original / wavelength`` (the scaling of Llama 3.1)."""
    factor: float
    low: float
    high: float
    original: float

    def apply(self, freqs: list, dims: int, base: float) -> list:
        out = []
        for f in freqs:
            turns = self.original * f / (2.0 * math.pi)           # original / wavelength
            if turns > self.high:
                out.append(f)
            elif turns < self.low:
                out.append(f / self.factor)
            else:
                keep = (turns - self.low) / (self.high - self.low)
                out.append(f * (keep + (1.0 - keep) / self.factor))
        return out

    def amplitude(self) -> float:
        return 1.0


@dataclass(frozen=True)
class RampScaling:
    """YaRN: pairs that turn more than ``fast`` times within ``original`` positions keep their frequency, those that turn less
    than ``slow`` times have it divided by ``factor``, with a linear ramp over the pair index between; cosine and sine grow
    by ``0.1 ln(factor) + 1``."""
    factor: float
    original: float
    fast: float
    slow: float

    def apply(self, freqs: list, dims: int, base: float) -> list:
        def pair_turning(times: float) -> float:
            return dims * math.log(self.original / (2.0 * math.pi * times)) / (2.0 * math.log(base))
        lo = max(math.floor(pair_turning(self.fast)), 0)
        hi = min(math.ceil(pair_turning(self.slow)), dims - 1)
        width = max(hi - lo, 0.001)
        out = []
        for i, f in enumerate(freqs):
            slowed = min(max((i - lo) / width, 0.0), 1.0)
            out.append(f * (slowed / self.factor + 1.0 - slowed))
        return out

    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0


@dataclass(frozen=True)
class RotaryConfig:
    """Rotation of the first ``dims`` entries of a head.  ``pairing``: ``"half"`` turns entry ``i`` with ``i + dims/2``,
    ``"next"`` entry ``2i`` with ``2i + 1``."""
    dims: int
    base: float
    pairing: str = "half"
    scaling: Optional[Union[BandScaling, RampScaling]] = None

    def __post_init__(self):
        if self.dims < 0 or self.dims % 2:
            raise ValueError(f"rotated dimensions must be even, got {self.dims}")
        if self.pairing not in ("half", "next"):
            raise ValueError(f"unknown pairing {self.pairing!r}")

    def frequencies(self) -> list:
        """Radians per position of the ``dims / 2`` pairs."""
        plain = [float(self.base) ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        return plain if self.scaling is None else self.scaling.apply(plain, self.dims, float(self.base))

    def amplitude(self) -> float:
        """Factor on cosine and sine."""
        return 1.0 if self.scaling is None else self.scaling.amplitude()
