"""Rotary position encodings.

``rotary_half``: pair (i, i + d/2), i < d/2, of the first ``rotary_dim`` = d elements of a head:
f_i = theta^(-2i/d), a = pos * f_i in float32,
x'_i = x_i cos a - x_{i+d/2} sin a,  x'_{i+d/2} = x_i sin a + x_{i+d/2} cos a
(reference: kernels/src/rope_kernel_cpu.cpp:127-141 for the table,
kernels/src/rope_kernel_cuda.cu:228-261 for the rotation; it always rotates the whole
head).  The frequencies are computed once on the host in float64 and rounded to
float32; the angle, sine and cosine are computed per token of the step, once per step for
all layers with the same frequencies (``step_table``), so there is no table whose length
bounds the context.

``rotary_pairs``: pair (2i, 2i + 1) of the first ``rotary_dim`` elements, the same angles.

Both take ``scaling`` (factor, low, high, original), which slows the frequencies that make few turns within the
``original`` length and leaves the fast ones alone (the scheme of Llama 3.1): with the wavelength l = 2 pi / f, f stays
where l < original / high, becomes f / factor where l > original / low, and between the two is the mean of both weighted
by how far original / l lies from ``low`` to ``high``.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

from .. import ops
from .registry import register
from .spec import ParamSpec


def scaled_frequencies(freq: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """``freq`` (float64) with the slow ones divided by ``factor``, the fast ones as they are and a blend between."""
    turns = original * freq / (2.0 * math.pi)                 # within the original length: original / wavelength
    share = ((turns - low) / (high - low)).clamp(0.0, 1.0) if high != low else (turns >= low).to(freq.dtype)
    return (1.0 - share) * freq / factor + share * freq


@register("position", "rotary_half")
class RotaryHalf:
    pairs = False          # whether elements 2i and 2i + 1 turn together rather than i and i + d/2

    def __init__(self, head_dim: int, theta: float, dtype: torch.dtype, device,
                 rotary_dim: Optional[int] = None, scaling: Optional[Dict[str, float]] = None):
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim if rotary_dim is not None else head_dim)
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and within head_dim {head_dim}")
        self.theta = float(theta)
        half = self.rotary_dim // 2
        idx = torch.arange(half, dtype=torch.float64)
        freq = self.theta ** (-2.0 * idx / self.rotary_dim)
        self.scaling = None
        if scaling is not None:
            self.scaling = tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))
            if not self.scaling[0] > 0.0 or not self.scaling[3] > 0.0:
                raise ValueError(f"a scaling needs a positive factor and original length, got {scaling}")
            freq = scaled_frequencies(freq, *self.scaling)
        self.inv_freq = freq.to(torch.float32).to(device)

    @classmethod
    def param_specs(cls, **params) -> Dict[str, ParamSpec]:
        return {}

    def load(self, tensors) -> None:
        pass

    def fused_rotary(self) -> Tuple[torch.Tensor, int]:
        return self.inv_freq, self.rotary_dim

    def step_table(self, ctx) -> Optional[torch.Tensor]:
        """Cosines and sines of this step's positions, [tokens, 2, rotary_dim / 2] float32, made by the
        first layer of the step that asks and kept in the step's context for the others."""
        memo = getattr(ctx, "memo", None)
        if memo is None or not self.inv_freq.is_cuda:
            return None
        key = ("rotary_half", self.theta, self.rotary_dim, self.scaling)
        table = memo.get(key)
        if table is None:
            table = memo[key] = ops.rope_table(ctx.positions, self.inv_freq)
        return table


@register("position", "rotary_pairs")
class RotaryPairs(RotaryHalf):
    """The same rotation of neighbouring elements, for attention parts whose norm kernel turns pairs."""
    pairs = True

    def step_table(self, ctx) -> Optional[torch.Tensor]:
        return None        # the kernels that read a step's table turn halves
