"""Rotary tables for pairs (i, i + dims / 2), with optional interpolation of the frequencies: YaRN (scaling with fast and slow)
or by bands of wavelengths (scaling with low and high)."""

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


def banded_frequencies(dims: int, base: float, scaling: dict) -> Tensor:
    """Angle per position of each of the dims / 2 pairs, fp64. scaling: factor, original, low, high. A pair that turns more than
    `high` times over the original context keeps its frequency, one that turns less than `low` times is divided by the factor,
    and those between mix the two in proportion to their turns."""
    freqs, _ = yarn_frequencies(dims, base, None)
    turns = freqs * (float(scaling["original"]) / (2.0 * math.pi))
    low, high = float(scaling["low"]), float(scaling["high"])
    slowed = freqs / float(scaling["factor"])
    share = ((turns - low) / (high - low)) if high > low else torch.zeros_like(turns)
    mixed = torch.where(turns < low, slowed, slowed * (1.0 - share) + freqs * share)
    return torch.where(turns > high, freqs, mixed)


def frequencies(dims: int, base: float, scaling: "dict | None") -> tuple[Tensor, float]:
    """(angle per position of each pair, factor of cos and sin) for either kind of scaling, or none."""
    if scaling and "low" in scaling:
        return banded_frequencies(dims, base, scaling), 1.0
    return yarn_frequencies(dims, base, scaling)


def half_tables(positions: int, dims: int, base: float, scaling: "dict | None", padded: int,
                device: "torch.device | str") -> tuple[Tensor, Tensor]:
    """cos, sin fp32 (positions, padded / 2), evaluated in fp64 and rounded once; pairs past dims / 2 do not turn."""
    freqs, factor = frequencies(dims, base, scaling)
    angle = torch.zeros((positions, padded // 2), dtype=torch.float64)
    angle[:, :dims // 2] = torch.arange(positions, dtype=torch.float64)[:, None] * freqs
    return (angle.cos() * factor).float().to(device), (angle.sin() * factor).float().to(device)
