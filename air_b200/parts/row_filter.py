"""What stands between a norm and the part that reads its rows."""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import TensorSpec
from .base import RowFilter, SlotState
from .registry import register_row_filter


@register_row_filter("residual_conv")
class ResidualConvolution(RowFilter):
    """x_t + sum_j w[:, j] x_(t - taps + 1 + j): a causal convolution over time on every channel, added to its input.  The
    last taps - 1 inputs are the request's state (32-bit, zeros at its start).  params: size, taps.  Tensor: <prefix>
    [size, taps] (the prefix is the tensor's whole name).  32-bit; the sum is rounded to the compute dtype once."""

    graph_safe = True

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        self.size, self.taps = int(spec["size"]), int(spec["taps"])

    def cache_needs(self):
        return (SlotState((self.taps - 1, self.size)),) if self.taps > 1 else ()

    def tensor_specs(self):
        return [TensorSpec(self.prefix, (self.size, self.taps), wide=True, std=0.3)]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        self.weight = tensors[self.prefix].to(torch.float32).t().contiguous()       # [taps, size]

    def _state(self, cache):
        return cache[0].state if self.taps > 1 else None

    def single_tokens(self, ctx, cache):
        return (self.weight, self._state(cache), ctx.token_seq) if ctx.all_decode else None

    def forward(self, x, ctx, cache):
        out = torch.empty(x.shape, dtype=self.rt.dtype, device=x.device)
        return ops.residual_conv(x, self.weight, self._state(cache), out, ctx.q_start, ctx.slots, ctx.max_q_len)
