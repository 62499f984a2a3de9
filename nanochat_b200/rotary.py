"""Rotary tables for pairs (i, i + dims / 2), with optional YaRN interpolation of the frequencies."""

import math

import torch
from torch import Tensor


def yarn_frequencies(dims: int, base: float, scaling: "dict | None") -> tuple[Tensor, float]:
    """(angle per position of each of the dims / 2 pairs, fp64; factor of both cos and sin). scaling: None, or factor,
    original (the context the base frequencies were made for), fast and slow (turns over that context above which a pair
    keeps its frequency, and below which it is divided by the factor; a linear ramp over the pair index in between)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    freqs = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / dims)
    if not scaling:
        return freqs, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_with_turns(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_with_turns(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_with_turns(float(scaling["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freqs / factor * ramp + freqs * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def half_tables(positions: int, dims: int, base: float, scaling: "dict | None", padded: int,
                device: "torch.device | str") -> tuple[Tensor, Tensor]:
    """cos, sin fp32 (positions, padded / 2), evaluated in fp64 and rounded once; pairs past dims / 2 do not turn."""
    freqs, factor = yarn_frequencies(dims, base, scaling)
    angle = torch.zeros((positions, padded // 2), dtype=torch.float64)
    angle[:, :dims // 2] = torch.arange(positions, dtype=torch.float64)[:, None] * freqs
    return (angle.cos() * factor).float().to(device), (angle.sin() * factor).float().to(device)
