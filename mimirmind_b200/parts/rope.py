"""Rotary position encoding, split-half pairing, with theta and the rotated width as parameters.

Pairs are ``(i, i + half)``; ``angle = pos · theta^(−2i/dim)``;
``x'_i = x_i cos − x_{i+half} sin``, ``x'_{i+half} = x_i sin + x_{i+half} cos``
(src/compute/Rope.cpp:23-41).  Applied to q and k after their bias, never to v
(src/runtime/arch/Qwen2Backend.cpp:369-375).  Angles are computed in fp32 on the device.
"""
from __future__ import annotations

import math
from typing import Any, Mapping, Optional, Tuple

import torch

from ..config.spec import PartSpec
from ..registry import POSITION_ENCODINGS
from .base import NativeDesc, PositionEncoding, Runtime, WeightView


def exact_frequencies(base: float, dims: int, scaling: Optional[Mapping[str, Any]] = None) -> Tuple[torch.Tensor, float]:
    """``base^(-2i/dims)`` for ``i < dims/2`` in float64, and what multiplies cos and sin.  With ``scaling`` (``factor``,
    ``original``, ``fast``, ``slow``) YaRN's interpolation: the pair that turns ``t`` times over ``original`` positions is number
    ``dims ln(original / (2 pi t)) / (2 ln base)``; up to the one of ``fast`` turns frequencies stay, from the one of ``slow`` turns on
    they are divided by ``factor``, between them in proportion; cos and sin are multiplied by ``0.1 ln(factor) + 1``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / dims)
    if scaling is None:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def number(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(number(float(scaling["fast"]))), 0)
    last = min(math.ceil(number(float(scaling["slow"]))), dims - 1)
    ramp = ((i - first) / max(last - first, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


@POSITION_ENCODINGS.register("rotary_half")
class RotaryHalf(PositionEncoding):
    """spec params: theta, rotary_dim (leading dims of each head that rotate)."""

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.theta = float(spec["theta"])
        self.rotary_dim = int(spec["rotary_dim"])
        if self.rotary_dim % 2:
            raise ValueError("rotary_dim must be even")

    def fused_rotary(self) -> Optional[Tuple[int, float]]:
        return self.rotary_dim, self.theta

    def native(self):
        if type(self) is not RotaryHalf:
            return None
        return NativeDesc("rotary_half", {"theta": self.theta, "rotary_dim": self.rotary_dim})


@POSITION_ENCODINGS.register("none")
class NoPositionEncoding(PositionEncoding):
    """No encoding: the fused kernel is told to rotate nothing."""

    def fused_rotary(self) -> Optional[Tuple[int, float]]:
        return 0, 1.0

    def native(self):
        return NativeDesc("none") if type(self) is NoPositionEncoding else None


@POSITION_ENCODINGS.register("rotary_pairs")
class RotaryPairs(PositionEncoding):
    """Rotation of adjacent pairs: dimensions ``2i`` and ``2i+1`` (``i < dims/2``) of every head turn by
    ``angle = pos * base^(-2i/dims)``: ``(u, v) -> (u cos - v sin, v cos + u sin)``; dimensions from ``dims`` on pass
    unchanged.  The frequencies are made once in float64 and kept as an fp32 table; the angle is an fp32 product.

    spec params: base, dims."""

    def __init__(self, spec: PartSpec, weights: WeightView, rt: Runtime):
        super().__init__(spec, weights, rt)
        self.base, self.dims = float(spec["base"]), int(spec["dims"])
        if self.dims % 2 or self.dims < 0:
            raise ValueError("rotary_pairs: dims must be even")
        i = torch.arange(max(1, self.dims // 2), dtype=torch.float64)
        self.inv_freq = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / max(1, self.dims)).to(torch.float32).to(rt.device)

    def pair_rotation(self) -> Tuple[int, "object"]:
        """(dims, fp32 frequency table) for kernels that rotate adjacent pairs themselves."""
        return self.dims, self.inv_freq
