"""A short causal convolution over time between a norm and its mixer."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import InputFilter, StateCacheSpec, TensorSpec
from .registry import register_part


class CausalConvolution(InputFilter):
    """``h + conv(h)``, per channel c and row t ``conv(h)[t, c] = sum_j w[c, j] h[t - (taps - 1) + j, c]`` (zeros before the
    sequence's start, no bias).  The tensor ``name`` is [width, taps], the last column the current token's; it is held in
    float32, and so are the inputs.  State per request: the last ``taps - 1`` inputs."""

    def __init__(self, size: int, taps: int, name: str = "conv"):
        if taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.size, self.taps, self.name = int(size), int(taps), name

    def tensor_specs(self, available=None):
        return {self.name: TensorSpec((self.size, self.taps), kind="vector")}

    def load(self, fetch, ctx):
        self.ctx = ctx
        self.weight = fetch(self.name).float().t().contiguous()           # [taps, width]

    def cache_spec(self):
        return StateCacheSpec((self.taps - 1, self.size)) if self.taps > 1 else None

    def forward(self, h32, batch, cache):
        out = torch.empty(h32.shape, dtype=self.ctx.act_dtype, device=h32.device)
        ops.causal_conv_add(h32, self.weight, batch, cache.state if self.taps > 1 else None, out)
        return out


register_part("input_filter", "causal_convolution", CausalConvolution)
