"""Rotary frequencies: scaling variants, and the per-batch table of models with per-layer mixers."""
from __future__ import annotations

import math

import torch

from ... import ops
from .config import RopeScaling, RotarySpec


def rope_frequencies(rot: int, theta: float, scaling: RopeScaling) -> tuple[torch.Tensor, float]:
    """Inverse rotary frequencies (double precision) with linear / llama3 / YaRN scaling, and the attention factor.
    (Reference: src/HartsyInference.Core/Rope/RopeFrequencyBuilder.cs, RopeScaling.cs.)"""
    inv = theta ** (-torch.arange(0, rot, 2, dtype=torch.float64) / rot)
    attn_factor = 1.0
    if scaling.kind == "linear":
        inv = inv / scaling.factor
    elif scaling.kind == "llama3":
        low = scaling.original_max_position / scaling.low_freq_factor
        high = scaling.original_max_position / scaling.high_freq_factor
        wavelen = 2 * math.pi / inv
        smooth = ((scaling.original_max_position / wavelen) - scaling.low_freq_factor) / (
            scaling.high_freq_factor - scaling.low_freq_factor)
        scaled = torch.where(wavelen > low, inv / scaling.factor, inv)
        mid = (wavelen <= low) & (wavelen >= high)
        scaled = torch.where(mid, (1 - smooth) * inv / scaling.factor + smooth * inv, scaled)
        inv = scaled
    elif scaling.kind == "yarn":
        def corr_dim(n_rot):
            return (rot * math.log(scaling.original_max_position / (n_rot * 2 * math.pi))) / (2 * math.log(theta))
        lo, hi = corr_dim(scaling.beta_fast), corr_dim(scaling.beta_slow)
        if scaling.truncate:
            lo, hi = math.floor(lo), math.ceil(hi)
        lo, hi = max(lo, 0), min(hi, rot // 2 - 1)
        ramp = ((torch.arange(rot // 2, dtype=torch.float64) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
        mask = 1 - ramp
        inv = inv / scaling.factor * (1 - mask) + inv * mask
        attn_factor = scaling.attn_factor * (0.1 * math.log(scaling.factor) + 1.0) if scaling.factor > 1 else 1.0
    return inv, attn_factor


def build_inv_freq(rot: int, theta: float, scaling: RopeScaling, device) -> tuple[torch.Tensor, float]:
    """:func:`rope_frequencies` in fp32 on ``device``, and the attention factor."""
    inv, attn_factor = rope_frequencies(rot, theta, scaling)
    return inv.to(torch.float32).to(device), attn_factor


class Rotary:
    """One rotation of a model with per-layer mixers: its frequencies as sums of two floats, and the table of cosines and
    sines of a batch, computed once for all layers that turn alike."""

    def __init__(self, spec: RotarySpec, device):
        self.spec = spec
        f, factor = rope_frequencies(spec.dims, spec.base, spec.scaling)
        if factor != 1.0:
            raise ValueError(f"rotary scaling '{spec.scaling.kind}' changes the attention scale, which per-layer mixers state themselves")
        hi = f.to(torch.float32)
        self.hi, self.lo = hi.to(device), (f - hi.double()).to(torch.float32).to(device)

    def table(self, batch) -> torch.Tensor:
        if batch.plan is None:
            batch.plan = {}
        key = ("rope", self.spec)
        if key not in batch.plan:
            batch.plan[key] = ops.rope_table(batch.positions, self.hi, self.lo)
        return batch.plan[key]
