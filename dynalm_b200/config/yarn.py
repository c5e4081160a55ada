"""YaRN: rotary frequencies stretched for positions beyond the range a model was trained on."""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Tuple

from ..errors import InvalidArgument
from .reader import KeyReader


@dataclass(frozen=True)
class YarnStretch:
    """Frequencies that turn more than `fast` times over `original` positions are kept, those that turn fewer than `slow`
    times are divided by `factor`, a linear ramp over the pairs lies in between; the rotated vectors grow by
    0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    def divisors(self, base: float, dims: int) -> Tuple[float, ...]:
        """What the frequency of every pair is divided by."""
        def pair_of(turns: float) -> float:
            return dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo = max(math.floor(pair_of(self.fast)), 0)
        hi = min(math.ceil(pair_of(self.slow)), dims - 1)
        out = []
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(1.0 / (ramp / self.factor + (1.0 - ramp)))
        return tuple(out)

    @property
    def magnitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    @classmethod
    def read(cls, sc: KeyReader, base: float) -> "YarnStretch":
        """From a `scaling` object with factor, original, fast and slow; `base` is the rotation's."""
        s = cls(sc.float_or("factor", 1.0), sc.float_or("original", 0.0), sc.float_or("fast", 32.0), sc.float_or("slow", 1.0))
        for name, value in (("factor", s.factor), ("original", s.original), ("fast", s.fast), ("slow", s.slow)):
            if not value > 0:
                raise InvalidArgument(f"{sc.where}: '{name}' must be positive")
        if base == 1.0:
            raise InvalidArgument(f"{sc.where}: a rotation of base 1 cannot be stretched")
        return s
