"""A block whose sublayers read the residual stream as it is and are normed on their way back into it:

    x <- x + scale * norm1(mixer(x));   x <- x + scale * norm2(feed_forward(x))      (the second line may be absent)

``residual_scale`` is one constant for both.  The norms are RMS norms.  What follows a sublayer is one launch: the norm of its
output, the sum into the 32-bit residual, and the new rows in the activation type for the sublayer that reads them next
(csrc/gated_ops.cu).
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import ops
from torchinferno_b200.parts.base import Block, LayerContext, Part, PartSpec, ResidualStream, build_part, register_part
from torchinferno_b200.parts.norm import RMSNorm


def _spec(value: PartSpec | Mapping | None) -> PartSpec | None:
    return value if value is None or isinstance(value, PartSpec) else PartSpec(**value)


class PostNormBlock(Block):
    def __init__(self, *, mixer: PartSpec, mixer_norm: PartSpec, feed_forward: PartSpec | None = None,
                 feed_forward_norm: PartSpec | None = None, residual_scale: float = 1.0,
                 dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if (feed_forward is None) != (feed_forward_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        self.specs = {"mixer": _spec(mixer), "mixer_norm": _spec(mixer_norm), "feed_forward": _spec(feed_forward),
                      "feed_forward_norm": _spec(feed_forward_norm)}
        self.mixer = build_part("mixer", self.specs["mixer"], dtype=dtype, device=device)
        self.mixer_norm = build_part("norm", self.specs["mixer_norm"], dtype=dtype, device=device)
        self.feed_forward = self.feed_forward_norm = None
        if feed_forward is not None:
            self.feed_forward = build_part("feed_forward", self.specs["feed_forward"], dtype=dtype, device=device)
            self.feed_forward_norm = build_part("norm", self.specs["feed_forward_norm"], dtype=dtype, device=device)
        for norm in (self.mixer_norm, self.feed_forward_norm):
            if norm is not None and not isinstance(norm, RMSNorm):
                raise ValueError(f"this block fuses RMS norms with the sums behind them; got {type(norm).__name__}")
        self.residual_scale = float(residual_scale)

    def named_parts(self) -> list[tuple[str, Part]]:
        return [(self.specs[key].prefix, getattr(self, key)) for key in ("mixer_norm", "mixer", "feed_forward_norm", "feed_forward")
                if self.specs[key] is not None]

    def _back(self, stream: ResidualStream, y: torch.Tensor, norm: RMSNorm) -> None:
        residual = stream.residual
        copy = None if stream.dtype == torch.float32 else torch.empty(residual.shape, dtype=stream.dtype, device=residual.device)
        ops.unit_norm_add(residual, y, norm.weight, norm.eps, self.residual_scale, copy)
        stream.activation_copy = copy

    def forward(self, stream: ResidualStream, ctx: LayerContext) -> None:
        self._back(stream, self.mixer.forward(stream.rows(), ctx), self.mixer_norm)
        if self.feed_forward is not None:
            self._back(stream, self.feed_forward.forward(stream.rows(), ctx), self.feed_forward_norm)


register_part("block", "postnorm", PostNormBlock)
