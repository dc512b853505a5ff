"""The arrangement of parts in one layer.

Pre-norm block (src/torchinferno/models/llama3/pipeline.py:190-198):
    h = h + mixer(norm1(h));  h = h + feed_forward(norm2(h))      (the second line is absent in a layer without a feed-forward)
With ``mixer_input`` / ``feed_forward_input`` (parts of category ``input_stage``) a sublayer reads what that stage makes of the
normed rows, e.g. their sum with a short convolution over time; what the stages carry from step to step is the block's state.
The adds are left pending on the residual stream so the next norm (of this
block, of the next block or the final one) does them in its own pass
(src/torchinferno/models/llama3/tensor_parallel.py:7430-7435).
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import gemm, native_block
from torchinferno_b200.parts.base import (Block, LayerContext, Part, PartSpec, ResidualStream, StateSpec,
                                          build_part, register_part)


NATIVE_BLOCKS = True          # False: always the part-by-part sequence
_UNKNOWN = object()


def _spec(value: PartSpec | Mapping | None) -> PartSpec | None:
    return value if value is None or isinstance(value, PartSpec) else PartSpec(**value)


class PreNormBlock(Block):
    def __init__(self, *, mixer: PartSpec, feed_forward: PartSpec | None, mixer_norm: PartSpec,
                 feed_forward_norm: PartSpec | None, mixer_input: PartSpec | None = None,
                 feed_forward_input: PartSpec | None = None, dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if (feed_forward is None) != (feed_forward_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        if feed_forward is None and feed_forward_input is not None:
            raise ValueError("there is no feed-forward to make an input for")
        self.specs = {"mixer": _spec(mixer), "feed_forward": _spec(feed_forward),
                      "mixer_norm": _spec(mixer_norm), "feed_forward_norm": _spec(feed_forward_norm),
                      "mixer_input": _spec(mixer_input), "feed_forward_input": _spec(feed_forward_input)}
        self.mixer = build_part("mixer", self.specs["mixer"], dtype=dtype, device=device)
        self.feed_forward = None if feed_forward is None else \
            build_part("feed_forward", self.specs["feed_forward"], dtype=dtype, device=device)
        self.mixer_norm = build_part("norm", self.specs["mixer_norm"], dtype=dtype, device=device)
        self.feed_forward_norm = None if feed_forward is None else \
            build_part("norm", self.specs["feed_forward_norm"], dtype=dtype, device=device)
        self.mixer_input = None if mixer_input is None else \
            build_part("input_stage", self.specs["mixer_input"], dtype=dtype, device=device)
        self.feed_forward_input = None if feed_forward_input is None else \
            build_part("input_stage", self.specs["feed_forward_input"], dtype=dtype, device=device)
        self._native = _UNKNOWN
        self._native_generation = -1

    def named_parts(self) -> list[tuple[str, Part]]:
        parts = [(self.specs["mixer_norm"].prefix, self.mixer_norm), (self.specs["mixer"].prefix, self.mixer)]
        if self.feed_forward is not None:
            parts += [(self.specs["feed_forward_norm"].prefix, self.feed_forward_norm),
                      (self.specs["feed_forward"].prefix, self.feed_forward)]
        parts += [(self.specs[name].prefix, stage) for name, stage in self._input_stages()]
        return parts

    def _input_stages(self) -> list[tuple[str, Part]]:
        return [(name, stage) for name, stage in (("mixer_input", self.mixer_input), ("feed_forward_input", self.feed_forward_input))
                if stage is not None]

    def block_state_spec(self) -> StateSpec | None:
        floats = sum(stage.state_floats() for _, stage in self._input_stages())
        return StateSpec((floats,), torch.float32) if floats else None

    @property
    def capturable(self) -> bool:
        return all(stage.capturable for _, stage in self._input_stages())

    def _read(self, stream: ResidualStream, norm, stage, ctx: LayerContext, state_off: int) -> torch.Tensor:
        return stream.normed(norm) if stage is None else stage.forward(stream, norm, ctx, state_off)

    def forward(self, stream: ResidualStream, ctx: LayerContext) -> None:
        if self._native is _UNKNOWN or self._native_generation != gemm.generation():
            # (decided at the first use, when the weights are bound, and again whenever a weight was bound or a
            # kernel choice changed since: a block of the built-in parts in bfloat16 is issued as one call into
            # the CUDA library, the same kernels in the same order)
            self._native = native_block.block_weights(self) if NATIVE_BLOCKS else None
            self._native_generation = gemm.generation()
        if self._native is not None and ctx.kv is not None and ctx.kv.writes and ctx.batch is not None:
            window = self.mixer.window if self.mixer.window is not None else ctx.kv.window
            native_block.run_block(self._native, stream, ctx, window)
            return
        stream.add(self.mixer.forward(self._read(stream, self.mixer_norm, self.mixer_input, ctx, 0), ctx))
        if self.feed_forward is not None:
            behind = 0 if self.mixer_input is None else self.mixer_input.state_floats()
            stream.add(self.feed_forward.forward(
                self._read(stream, self.feed_forward_norm, self.feed_forward_input, ctx, behind), ctx))


register_part("block", "prenorm", PreNormBlock)
