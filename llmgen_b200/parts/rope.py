"""Rotary position encoding: the cos/sin tables its mixer's kernel reads."""
from __future__ import annotations

import math
from typing import Dict, Tuple

import torch

from .base import Part
from .registry import register_position
from .spec import RopeSpec

_TABLES: Dict[Tuple, Tuple[torch.Tensor, torch.Tensor]] = {}


def scale_by_wavelength(inv: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequencies (float64) scaled by their wavelength l = 2 pi / f: unchanged where l < original / high, divided by
    `factor` where l > original / low, and between the two (1 - s) f / factor + s f with
    s = (original / l - low) / (high - low)."""
    if high <= low:
        raise ValueError(f"rotary scaling: high {high} must exceed low {low}")
    wave = 2.0 * math.pi / inv
    s = (original / wave - low) / (high - low)
    blended = (1.0 - s) * inv / factor + s * inv
    return torch.where(wave < original / high, inv, torch.where(wave > original / low, inv / factor, blended))


def scale_by_place(inv: torch.Tensor, theta: float, factor: float, original: float, fast: float, slow: float) -> torch.Tensor:
    """Frequencies (float64, pair i of rotary_dim / 2) scaled by the pair's place: f where the pair turns at least `fast` times
    within `original` positions, f / factor where at most `slow` times, and a blend in between (YaRN)."""
    half = inv.numel()
    dims = 2 * half

    def place(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))

    lo, hi = max(math.floor(place(fast)), 0), min(math.ceil(place(slow)), dims - 1)
    ramp = ((torch.arange(half, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return inv / factor * ramp + inv * (1.0 - ramp)


class Rope(Part):
    """cos/sin of pos / theta^(2i / rotary_dim), i in [0, rotary_dim/2), for every position:
    computed once on the host in float64 and kept as float32 [max_positions, rotary_dim/2]
    (the reference computes inverse frequencies and angles in f64 and stores f32 rows whose two
    halves are equal, src/backend/cpu/rope.zig:47-75; only one half is kept here).  Layers
    with the same spec share one pair of tables.  `spec.scaling` rescales the frequencies by their wavelength first
    (`scale_by_wavelength`), `spec.yarn` by the pair's place (`scale_by_place`; both tables are then multiplied by
    0.1 ln(factor) + 1)."""

    def __init__(self, spec: RopeSpec, weights, dtype, device):
        self.spec = spec
        scaling = tuple(float(v) for v in spec.scaling) if getattr(spec, "scaling", None) is not None else None
        yarn = tuple(float(v) for v in spec.yarn) if getattr(spec, "yarn", None) is not None else None
        if scaling is not None and yarn is not None:
            raise ValueError("rotary encoding: frequencies are scaled by wavelength or by place, not both")
        key = (spec.rotary_dim, float(spec.theta), spec.max_positions, scaling, yarn, str(device))
        if key not in _TABLES:
            half = spec.rotary_dim // 2
            inv = 1.0 / torch.pow(torch.tensor(float(spec.theta), dtype=torch.float64),
                                  torch.arange(0, half, dtype=torch.float64) * 2.0 / spec.rotary_dim)
            if scaling is not None:
                inv = scale_by_wavelength(inv, *scaling)
            amplitude = 1.0
            if yarn is not None:
                inv = scale_by_place(inv, float(spec.theta), *yarn)
                amplitude = 0.1 * math.log(yarn[0]) + 1.0
            ang = torch.arange(spec.max_positions, dtype=torch.float64)[:, None] * inv[None, :]
            _TABLES[key] = ((ang.cos() * amplitude).to(torch.float32).to(device).contiguous(),
                            (ang.sin() * amplitude).to(torch.float32).to(device).contiguous())
        self.cos, self.sin = _TABLES[key]
        self.rotary_dim = spec.rotary_dim
        self.pairing = spec.pairing
        self.max_positions = spec.max_positions

    def tables(self):
        return self.cos, self.sin


register_position("rope", Rope)
