"""Rotary position embedding as configurations give it."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional, Tuple


@dataclass
class RotaryConfig:
    """Rotary embedding of the first `dims` dimensions of a head, with YaRN scaling when `factor` is given."""
    base: float
    dims: int
    factor: Optional[float] = None
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    @staticmethod
    def parse(c: Optional[dict]) -> "RotaryConfig":
        if not c:
            return RotaryConfig(1.0, 0)
        s = c.get("scaling") or {}
        return RotaryConfig(float(c["base"]), int(c["dims"]), float(s["factor"]) if s else None, float(s.get("original", 0)),
                            float(s.get("fast", 0)), float(s.get("slow", 0)))

    def frequencies(self) -> Tuple[List[float], float]:
        """(angle per token of every pair, gain of cos and sin)."""
        n = self.dims
        freq = [self.base ** (-2.0 * i / n) for i in range(n // 2)]
        if self.factor is None:
            return freq, 1.0

        def pair_that_turns(times: float) -> float:          # how many turns a pair makes over the original context
            return n * math.log(self.original / (2.0 * math.pi * times)) / (2.0 * math.log(self.base))

        lo = max(math.floor(pair_that_turns(self.fast)), 0)
        hi = min(math.ceil(pair_that_turns(self.slow)), n - 1)
        width = max(hi - lo, 0.001)
        ramp = [min(max((i - lo) / width, 0.0), 1.0) for i in range(n // 2)]
        return [f / self.factor * r + f * (1.0 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(self.factor) + 1.0
