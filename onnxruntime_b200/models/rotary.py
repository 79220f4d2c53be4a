"""Rotary tables in fp32 (angles in float64) with the frequency rescalings of long-context models."""
from __future__ import annotations

import math
from typing import Any, Mapping, Tuple

import torch


def _three_bands(f: torch.Tensor, sc: Mapping[str, Any]) -> torch.Tensor:
    """Short wavelengths stay, long ones are stretched by ``factor``, a linear blend in between (Llama 3)."""
    wavelength = 2.0 * math.pi / f
    s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
    blend = (1.0 - s) * f / sc["factor"] + s * f
    return torch.where(wavelength < sc["original"] / sc["high"], f, torch.where(wavelength > sc["original"] / sc["low"], f / sc["factor"], blend))


def _yarn(f: torch.Tensor, rot: Mapping[str, Any]) -> Tuple[torch.Tensor, float]:
    """YaRN: pairs that turn more than ``fast`` times within the original length stay, those below ``slow`` turns are stretched
    by ``factor``, with a ramp over the pair index in between.  The second result multiplies cos and sin."""
    sc, dims, base = rot["scaling"], rot["dims"], float(rot["base"])

    def index(turns: float) -> float:
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index(sc["fast"])), 0), min(math.ceil(index(sc["slow"])), dims - 1)
    ramp = ((torch.arange(f.numel(), dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotary_tables(rot: Mapping[str, Any], rows: int, device="cpu") -> Tuple[torch.Tensor, torch.Tensor]:
    """cos / sin [rows, dims / 2] of positions 0 .. rows - 1.  ``rot``: base, dims and optionally "scaling" (factor, original and
    either low / high: three bands, or fast / slow: YaRN)."""
    half = rot["dims"] // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=torch.float64) / rot["dims"])
    sc, gain = rot.get("scaling"), 1.0
    if sc:
        if "fast" in sc:
            f, gain = _yarn(f, rot)
        else:
            f = _three_bands(f, sc)
    angles = torch.outer(torch.arange(rows, dtype=torch.float64), f)
    return (gain * angles.cos()).float().to(device), (gain * angles.sin()).float().to(device)
