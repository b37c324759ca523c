"""Learned absolute positions: a table row per position, added to the token embedding
(reference: crates/core/src/kernels/reference.rs:86-94).  The table's length bounds the
context (crates/core/src/stages/mod.rs:516-519)."""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from ..kernels import ops
from .base import TABLE, ParamSpec, PositionEncoding, register_position


@register_position("learned_absolute")
class LearnedAbsolutePositions(PositionEncoding):
    def __init__(self, n_positions: int, width: int):
        self.n_positions, self.width = int(n_positions), int(width)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("table", (self.n_positions, self.width), TABLE)]

    def additive_table(self) -> Optional[torch.Tensor]:
        return self.params["table"]

    def max_positions(self) -> Optional[int]:
        return self.n_positions


@register_position("rotary_pairs")
class RotaryPairs(PositionEncoding):
    """Rotary positions inside a mixer: of every query and key head the first ``dims`` values turn in pairs
    (2i, 2i + 1) (the interleaved layout) by the angle position * base^(-2i / dims); the other values pass.
    It has no parameters.  The frequencies are made in double precision on the host; the rotation itself is
    done by the mixer's own kernel between the projection and the cache (``kernels.ops.rope_append``), which asks
    this part for ``dims`` and ``freqs``."""

    def __init__(self, base: float, dims: int):
        if dims < 0 or dims % 2:
            raise ValueError(f"rotary_pairs: dims {dims} must be even and not negative")
        if dims and not base > 0.0:
            raise ValueError(f"rotary_pairs: base {base} must be positive")
        self.base, self.dims = float(base), int(dims)
        self.freqs: Optional[torch.Tensor] = None

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        if self.dims:
            i = torch.arange(self.dims // 2, dtype=torch.float64)
            self.freqs = (self.base ** (-2.0 * i / self.dims)).to(device)

    def on_qk(self, q, k, ctx) -> None:
        raise NotImplementedError("rotary_pairs turns queries and keys inside ops.rope_append, on the projection's "
                                  "32-bit output; a mixer that holds it calls that")


@register_position("sinusoidal")
class SinusoidalPositions(PositionEncoding):
    """Fixed sinusoidal positions added to the embedding: entry 2i of a row at position p gets
    sin(p * base^(-2i / width)), entry 2i + 1 the cosine of the same angle.  No parameters and no table: the
    frequencies are made in double precision on the host, and one kernel makes angle, sine and cosine in double
    precision from the row's position, so no length bounds the context."""

    def __init__(self, width: int, base: float = 10000.0):
        if width <= 0 or not base > 0.0:
            raise ValueError("sinusoidal: width and base must be positive")
        self.width, self.base = int(width), float(base)
        self.freqs: Optional[torch.Tensor] = None

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        i = torch.arange((self.width + 1) // 2, dtype=torch.float64)
        self.freqs = (self.base ** (-2.0 * i / self.width)).to(device)

    def on_embedding(self, x, ctx) -> None:
        ops.add_sinusoid(x, ctx.positions, self.freqs, ctx.n_rows)


@register_position("rotary_halves")
class RotaryHalves(RotaryPairs):
    """Rotary positions in the halves layout: of every query and key head the first ``dims`` values turn, value i
    paired with value i + dims / 2, by the angle position * base^(-2i / dims); the other values pass.  The rotation is
    done by the mixer's own kernel (``kernels.ops.wide_norm_rope_append``, ``kernels.ops.rope_halves``,
    ``kernels.ops.norm_rope_maps_append``).

    ``scaling`` (YaRN: factor, original, fast, slow) stretches the wavelengths for sequences longer than the ``original``
    length: with index(t) the index whose wave turns t times in that length, frequencies below lo =
    max(floor(index(fast)), 0) stay, those above hi = min(ceil(index(slow)), dims - 1) are divided by ``factor``, in
    between a ramp over the indices mixes the two; cosine and sine are multiplied by ``amplitude`` = 0.1 ln(factor) + 1
    (mixers whose kernel takes no amplitude refuse a scaled encoding)."""

    layout = "halves"

    def __init__(self, base: float, dims: int, scaling: Optional[dict] = None):
        super().__init__(base, dims)
        #: what cosine and sine are multiplied by
        self.amplitude = 1.0
        self.scaling = dict(scaling) if scaling else None
        if self.scaling is not None:
            missing = {"factor", "original", "fast", "slow"} - set(self.scaling)
            if missing or not all(float(self.scaling[k]) > 0.0 for k in ("factor", "original", "fast", "slow")):
                raise ValueError("rotary_halves: scaling needs positive factor, original, fast and slow")
            self.amplitude = 0.1 * math.log(float(self.scaling["factor"])) + 1.0

    def frequencies(self) -> List[float]:
        """The ``dims`` / 2 frequencies in double precision."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        sc = self.scaling
        if sc is None:
            return f

        def index(turns: float) -> float:
            # base^(-2i/dims) * original = 2 pi turns, solved for i
            return self.dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

        lo = max(math.floor(index(float(sc["fast"]))), 0)
        hi = min(math.ceil(index(float(sc["slow"]))), self.dims - 1)
        out = []
        for i, fi in enumerate(f):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(fi / float(sc["factor"]) * ramp + fi * (1.0 - ramp))
        return out

    def prepare(self, dtype, device) -> None:
        PositionEncoding.prepare(self, dtype, device)
        if self.dims:
            self.freqs = torch.tensor(self.frequencies(), dtype=torch.float64, device=device)
