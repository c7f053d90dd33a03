"""Position encodings for attention.

``RotaryEncoding`` restates src/forge_engine/qwen3.py:345-363: inv_freq_j =
1 / theta^(2j / rotary_dim) in 32-bit, angle = float(position) * inv_freq_j; the
rotation itself happens inside the fused q/k kernel.  Cosine and sine of a step's angles
are the same in every layer: ``table`` takes them once per step (in 32-bit, not rounded)."""

from __future__ import annotations

import math

import torch

from ..ops import native
from .base import BuildContext, PositionEncoding, register_part


class RotaryEncoding(PositionEncoding):
    graph_safe = True

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        if spec.rotary_dim % 2 or spec.rotary_dim > spec.head_dim:
            raise ValueError("rotary_dim must be even and at most head_dim")
        self.rotary_dim = spec.rotary_dim
        self.theta = float(spec.theta)
        # which elements form a pair is the business of the kernel that rotates; the angles
        # are the same either way
        self.interleaved = bool(getattr(spec, "interleaved", False))
        if self.interleaved:
            # theta^(-2j / rotary_dim) worked out in 64-bit and rounded once
            exponent = torch.arange(0, spec.rotary_dim, 2, dtype=torch.float64) / spec.rotary_dim
            self.inv_freq = (self.theta ** -exponent).float().to(ctx.device).contiguous()
        else:
            exponent = torch.arange(0, spec.rotary_dim, 2, dtype=torch.float32) / spec.rotary_dim
            self.inv_freq = (1.0 / (spec.theta**exponent)).to(ctx.device).contiguous()
        self.scaling = getattr(spec, "scaling", None)
        self.exact = bool(getattr(spec, "exact_frequencies", False))
        self.yarn = getattr(spec, "yarn", None)
        self.divisor = float(getattr(spec, "frequency_divisor", 1.0))
        self.amplitude = 1.0         # what cosine and sine are multiplied by
        if self.divisor <= 0:
            raise ValueError("frequencies are divided by a positive number")
        if self.scaling is not None or self.exact or self.yarn is not None or self.divisor != 1.0:
            exponent = torch.arange(0, spec.rotary_dim, 2, dtype=torch.float64) / spec.rotary_dim
            freq = self.theta ** -exponent / self.divisor
            if self.scaling is not None:
                freq = self.stretch(freq, self.scaling)
            if self.yarn is not None:
                freq, self.amplitude = self.ramp(freq, self.theta, spec.rotary_dim, self.yarn)
            self.inv_freq = freq.float().to(ctx.device).contiguous()

    @staticmethod
    def ramp(freq: torch.Tensor, theta: float, dims: int, yarn: tuple) -> tuple:
        """(frequencies, factor of cosine and sine) after blending every frequency with its
        ``factor``-th part by a ramp between the dimensions that turn ``fast`` and ``slow`` times
        within ``original`` positions (64-bit)."""
        factor, original, fast, slow = (float(v) for v in yarn)
        if min(factor, original, fast, slow) <= 0 or theta <= 0 or theta == 1:
            raise ValueError("frequency scaling needs positive numbers and a base other than 1")
        place = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))  # noqa: E731
        low, high = max(math.floor(place(fast)), 0), min(math.ceil(place(slow)), dims - 1)
        index = torch.arange(freq.numel(), dtype=torch.float64)
        part = ((index - low) / max(high - low, 0.001)).clamp(0.0, 1.0)
        return freq / factor * part + freq * (1.0 - part), 0.1 * math.log(factor) + 1.0

    @staticmethod
    def stretch(freq: torch.Tensor, scaling: tuple) -> torch.Tensor:
        """Frequencies stretched by wavelength l = 2 pi / f (64-bit in, 64-bit out): kept below
        original / high, divided by ``factor`` above original / low, and blended in between with
        s = (original / l - low) / (high - low) as (1 - s) f / factor + s f."""
        factor, low, high, original = (float(v) for v in scaling)
        if factor <= 0 or high <= low or original <= 0:
            raise ValueError("frequency scaling needs factor > 0, original > 0 and high > low")
        wave = 2.0 * math.pi / freq
        s = (original / wave - low) / (high - low)
        blended = (1.0 - s) * freq / factor + s * freq
        return torch.where(wave < original / high, freq, torch.where(wave > original / low, freq / factor, blended))

    def rotary(self):
        return self.inv_freq, self.rotary_dim

    def table(self, batch) -> torch.Tensor:
        """[tokens, rotary_dim / 2, 2] (cos, sin) of this step's angles; worked out by the
        first layer that asks and shared through the batch."""
        key = ("rotary", self.theta, self.rotary_dim, self.interleaved, self.scaling, self.exact, self.yarn, self.divisor)
        table = batch.shared.get(key)
        if table is None:
            table = torch.empty((batch.n_tokens, self.rotary_dim // 2, 2), dtype=torch.float32, device=self.inv_freq.device)
            native.rope_table(batch.positions, self.inv_freq, table, self.amplitude)
            batch.shared[key] = table
        return table


class NoPosition(PositionEncoding):
    graph_safe = True

    def __init__(self, spec, weights: dict, ctx: BuildContext) -> None:
        pass


register_part("rope", RotaryEncoding, replace=True)
register_part("none", NoPosition, replace=True)
