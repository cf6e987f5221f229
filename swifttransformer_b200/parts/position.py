"""Position encodings.

``LearnedPositions`` is OPT's: a table row per position, added to the token
embedding, stored with ``offset`` unused leading rows (the reference strips
them offline, scripts/lib/converter_lib.py:271, and adds the row in the
embedding kernel, src/csrc/kernel/embedding.cu:25-33).

An encoding that acts on queries and keys instead (rotary and the like) would
implement ``apply_qk``; the attention mixer calls it, when present, before the
keys go to the cache.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..weights.spec import TABLE, ParamSpec
from .base import POSITION_ENCODINGS, Part


class PositionEncoding(Part):
    def hidden_table(self) -> Optional[Tuple[torch.Tensor, int]]:
        """(table, offset) if this encoding is a row added to the hidden state, else None."""
        return None

    def max_positions(self) -> Optional[int]:
        return None

    # encodings of queries / keys override this: apply_qk(q, k, ctx) changes q [N, heads, head_dim] and
    # k [N, kv_heads, head_dim] in place (ctx.positions holds each token's position; -1 marks padding rows)
    apply_qk = None


@POSITION_ENCODINGS.register("none")
class NoPositions(PositionEncoding):
    def __init__(self, **_):
        pass


@POSITION_ENCODINGS.register("learned")
class LearnedPositions(PositionEncoding):
    def __init__(self, max_positions: int, width: int, offset: int, name: str):
        self._max, self.width, self.offset, self.name = max_positions, width, offset, name
        self.table: Optional[torch.Tensor] = None

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.name, (self._max + self.offset, self.width), TABLE)]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.name]

    def hidden_table(self):
        return self.table, self.offset

    def max_positions(self) -> int:
        return self._max

    def add_to(self, x: torch.Tensor, positions: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        return ops.add_positions(x, positions, self.table, self.offset, out)


@POSITION_ENCODINGS.register("rotary_pairs")
class RotaryPairs(PositionEncoding):
    """Rotation of queries and keys by position: of the first ``dims`` dimensions of a head, dimension 2i is paired
    with 2i+1 (neighbours, not halves) and the pair (u, v) at position p becomes (u cos a - v sin a, v cos a + u sin a)
    with a = p * base^(-2i/dims); the other dimensions pass unchanged.  The frequencies are computed once in double
    precision and kept as float32; the angle and its sine and cosine are float32 in the kernels.  A mixer that
    prepares its queries and keys in a kernel of its own takes ``inv_freq`` and ``dims`` from here."""

    neighbours = True

    def __init__(self, dims: int, base: float, scaling: Optional[Dict[str, float]] = None, **_):
        """``scaling``: None, or {"factor", "original", "fast", "slow"}, the YaRN stretch of the context: with
        turns(t) = dims * ln(original / (2 pi t)) / (2 ln base), the index at which a pair turns t times within
        ``original`` positions, pairs before floor(turns(fast)) keep their frequency, those after ceil(turns(slow)) turn
        ``factor`` times slower, a linear ramp lies between, and sine and cosine are multiplied by
        0.1 ln(factor) + 1 (``amplitude``).  Or {"factor", "original", "low", "high"}, a stretch by wavelength: with
        the wavelength l = 2 pi / f of a pair, pairs with l < original / high keep their frequency, those with
        l > original / low turn ``factor`` times slower, in between the two are mixed with the share
        (original / l - low) / (high - low) of the kept frequency; the amplitude stays 1."""
        if dims < 0 or dims % 2:
            raise ValueError(f"rotary dimensions must be even and not negative, got {dims}")
        self.dims, self.base = int(dims), float(base)
        self.scaling = dict(scaling) if scaling else None
        self._by_wavelength = bool(self.scaling) and "low" in self.scaling
        self.amplitude = 0.1 * math.log(self.scaling["factor"]) + 1.0 if self.scaling and not self._by_wavelength else 1.0
        self._tables: Dict[torch.device, torch.Tensor] = {}

    def frequencies(self) -> List[float]:
        """One frequency per pair, in double precision."""
        f = [math.pow(self.base, -2.0 * i / self.dims) for i in range(self.dims // 2)]
        if not self.scaling:
            return f
        s = self.scaling
        if self._by_wavelength:
            return [self._stretched(v) for v in f]
        turns = lambda t: self.dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), self.dims - 1)
        out = []
        for i, v in enumerate(f):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(v / s["factor"] * ramp + v * (1.0 - ramp))
        return out

    def _stretched(self, f: float) -> float:
        s, wavelength = self.scaling, 2.0 * math.pi / f
        if wavelength < s["original"] / s["high"]:
            return f
        if wavelength > s["original"] / s["low"]:
            return f / s["factor"]
        kept = (s["original"] / wavelength - s["low"]) / (s["high"] - s["low"])
        return (1.0 - kept) * f / s["factor"] + kept * f

    def inv_freq(self, device) -> torch.Tensor:
        device = torch.device(device)
        if device not in self._tables:
            self._tables[device] = torch.tensor(self.frequencies() or [0.0], dtype=torch.float64).to(torch.float32).to(device)
        return self._tables[device]


@POSITION_ENCODINGS.register("rotary_halves")
class RotaryHalves(RotaryPairs):
    """The same rotation with the other pairing: of the first ``dims`` dimensions of a vector, dimension i is paired
    with dimension i + dims/2 (the two halves, not neighbours), i = 0 .. dims/2 - 1, at the angle
    p * base^(-2i/dims).  A mixer that rotates in a kernel of its own takes ``inv_freq`` and ``dims`` from here."""

    neighbours = False
