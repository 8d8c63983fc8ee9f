"""Rotary position encoding: the per-step cos/sin tables.

Formula (upstream src/tinyserve/layers.py:61-65): ``inv_freq[i] = theta ** (-2i / rotary_dim)``
in float64, ``angle = position * inv_freq`` in float64, cos and sin taken in float64 and
rounded to float32. The rotation itself (pairs ``i`` and ``i + rotary_dim/2`` for the "half"
pairing, neighbours ``2i, 2i+1`` for "interleaved"; src/tinyserve/layers.py:84-91 has the
former) is applied by the mixer's fused kernel, which receives these tables. ``scaling``: the four
keys of the rule by wavelength below; ``factor, original, fast, slow`` for YaRN (``scale_yarn``, which also
puts a constant on cos and sin); or ``{"factor": f}`` alone for linear scaling (every frequency divided by ``f``).
"""

from __future__ import annotations

import math
from typing import Any

import torch

from ..kernels import ops
from .base import EVERY_STEP, PositionEncoding, Rotation, StepContext, register_position_encoding

RotaryTables = Rotation      # the step's position data of a rotary encoding is the rotation itself


def scale_by_wavelength(freq: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequency scaling by wavelength (the Llama 3.1 rule), in float64: with wavelength
    ``l = 2 pi / f``, ``f`` stays where ``l < original / high``, becomes ``f / factor`` where
    ``l > original / low``, and in between is ``(1 - s) f / factor + s f`` with
    ``s = (original / l - low) / (high - low)``."""
    if not (factor > 0 and high > low and original > 0):
        raise ValueError(f"rotary scaling needs factor > 0, high > low, original > 0; got {factor}, {low}, {high}, {original}")
    wavelength = 2.0 * math.pi / freq
    s = (original / wavelength - low) / (high - low)
    blended = (1.0 - s) * freq / factor + s * freq
    out = torch.where(wavelength > original / low, freq / factor, blended)
    return torch.where(wavelength < original / high, freq, out)


def scale_yarn(freq: torch.Tensor, dims: int, base: float, factor: float, original: float, fast: float, slow: float) -> torch.Tensor:
    """YaRN: pair i keeps its frequency where it turns more than ``fast`` times over ``original`` positions, has it
    divided by ``factor`` where it turns less than ``slow`` times, and moves between the two along a ramp over the
    pairs' indices (float64). The bounds are the indices at which a pair of ``base^(-2i/dims)`` turns that often,
    rounded outwards and kept inside ``0 .. dims - 1``."""
    if not (factor > 0 and original > 0 and fast > 0 and slow > 0 and base > 1):
        raise ValueError(f"YaRN needs positive factor, original, fast, slow and base > 1; got {factor}, {original}, {fast}, {slow}, {base}")

    def index(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), dims - 1)
    i = torch.arange(freq.shape[0], dtype=torch.float64)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp)


class RotaryEncoding(PositionEncoding):
    recordable = EVERY_STEP

    def __init__(self, head_dim: int, rotary_dim: int, theta: float, pairing: str = "half",
                 scaling: "dict[str, float] | None" = None) -> None:
        if rotary_dim % 2 or not 0 < rotary_dim <= head_dim:
            raise ValueError(f"rotary_dim={rotary_dim} must be even and at most head_dim={head_dim}")
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"pairing must be 'half' or 'interleaved', got {pairing!r}")
        self.head_dim, self.rotary_dim = int(head_dim), int(rotary_dim)
        self.theta, self.pairing = float(theta), pairing
        two_i = torch.arange(0, self.rotary_dim, 2, dtype=torch.float64)
        self._inv_freq_host = self.theta ** (-two_i / self.rotary_dim)
        self.scaling = None
        self.mult = 1.0                 # a constant on cos and sin
        if scaling and set(scaling) == {"factor", "original", "fast", "slow"}:
            values = [float(scaling[k]) for k in ("factor", "original", "fast", "slow")]
            self.scaling = ("yarn", *values)
            self._inv_freq_host = scale_yarn(self._inv_freq_host, self.rotary_dim, self.theta, *values)
            self.mult = 0.1 * math.log(values[0]) + 1.0
        elif scaling and set(scaling) == {"factor"}:
            # linear scaling: every frequency divided by the factor (positions stretched by it)
            if not float(scaling["factor"]) > 0:
                raise ValueError(f"rotary scaling factor must be positive, got {scaling['factor']}")
            self.scaling = ("linear", float(scaling["factor"]))
            self._inv_freq_host = self._inv_freq_host / self.scaling[1]
        elif scaling:
            self.scaling = tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))
            self._inv_freq_host = scale_by_wavelength(self._inv_freq_host, *self.scaling)
        self._inv_freq: torch.Tensor | None = None

    def key(self) -> Any:
        return ("rope", self.rotary_dim, self.theta, self.pairing, self.scaling)

    def prepare(self, ctx: StepContext) -> RotaryTables:
        dev = ctx.positions.device
        if self._inv_freq is None or self._inv_freq.device != dev:
            self._inv_freq = self._inv_freq_host.to(dev)
        half = self.rotary_dim // 2
        cos = ctx.arena.take_step((ctx.num_tokens, half), torch.float32)
        sin = ctx.arena.take_step((ctx.num_tokens, half), torch.float32)
        if self.mult == 1.0:
            ops.rope_tables(ctx.positions, self._inv_freq, cos, sin)
        else:
            ops.rope_tables(ctx.positions, self._inv_freq, cos, sin, self.mult)
        return RotaryTables(cos, sin, self.rotary_dim, self.pairing == "interleaved")


register_position_encoding("rope", RotaryEncoding)
