"""What a sublayer reads, when that is more than a norm of the residual stream.

``causal_conv``  h + conv(h), with h the normed rows: a short causal convolution over time on each channel, conv(h)_t = sum_j
                 w[:, j] h_(t - taps + 1 + j), rows before a sequence's start taken as zero.  No bias, no activation.  The last
                 taps - 1 rows h are the stage's state of a request (fp32, oldest first).

A step of single tokens behind an RMS norm is one launch: residual sum, norm, convolution and the move of the carried rows
(csrc/input_conv.cu); any other step is the norm's launch and one more.
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import ops
from torchinferno_b200.parts.base import InputStage, LayerContext, Norm, ResidualStream, WeightSpec, register_part
from torchinferno_b200.parts.norm import RMSNorm


class CausalConvInput(InputStage):
    capturable = True       # (state is read and written by the kernels through the slots array)

    def __init__(self, *, width: int, taps: int, weight_name: str = "conv", dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if taps < 1:
            raise ValueError("the convolution has at least one tap")
        self.width, self.taps, self.weight_name = int(width), int(taps), weight_name
        self.conv_weight: torch.Tensor | None = None

    def weight_specs(self) -> list[WeightSpec]:
        return [WeightSpec(self.weight_name, (self.width, self.taps), std=0.5 * self.taps ** -0.5, role="vector")]

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        self.conv_weight = weights[self.weight_name].to(torch.float32).t().contiguous()      # [taps, width]

    def state_floats(self) -> int:
        return (self.taps - 1) * self.width

    def forward(self, stream: ResidualStream, norm: Norm, ctx: LayerContext, state_off: int) -> torch.Tensor:
        batch, state = ctx.batch, ctx.block_state
        residual = stream.residual
        out = torch.empty(residual.shape, dtype=stream.dtype, device=residual.device)
        pending = stream.pending
        if (batch.max_q_len == 1 and batch.n_tokens == batch.n_entries and type(norm) is RMSNorm
                and (pending is None or (pending.dtype == stream.dtype and pending.is_contiguous()))):
            ops.norm_conv_step(pending, residual, norm.weight, norm.eps, self.conv_weight, state, state_off, batch.slots, out)
            stream.pending = None
            return out
        return ops.input_conv(stream.normed(norm), out, self.conv_weight, state, state_off, batch.q_start, batch.slots,
                              batch.n_entries, batch.max_q_len)


register_part("input_stage", "causal_conv", CausalConvInput)
