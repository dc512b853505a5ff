"""Grouped attention inside a sliding window that keeps the first tokens in sight, on convolved queries and keys.

q = W_q x and k = W_k x pass a causal convolution over time on every channel (``taps``; weights ``q.conv`` / ``k.conv`` [channels,
taps], the last column the current row's; zeros before a sequence's start); the values are k as it leaves the convolution (there is
no W_v).  With ``row_norm_eps`` the whole q row and the whole k row, all heads at once, are then divided by their root mean square
and multiplied by a weight per element (``q.norm`` / ``k.norm``), and both get the position encoding (``position``: rotary over
interleaved pairs, possibly on part of a head).  A query at i sees j <= i with i - j < ``window`` or j < ``keep_first``
(``window`` None: every earlier token); score = q . k * ``scale``; the softmax's denominator also holds exp(sink): a learned number per
head with ``sink="learned"``, 1 (a sink of 0) with ``sink="one"``, nothing with None.  The heads side by side are multiplied
element by element by sigmoid(W_g x) (``gate``) and projected by W_o.  Query head h reads key/value head h // (heads / kv_heads).

The last taps - 1 projected rows of q and k are the mixer's state of a request.  What lies between the input projections (one
product) and the scores is one kernel (csrc/conv_norm_append.cu); the attention is the windowed attention's
(csrc/pooled_window_attention.cu) with its first tokens kept.
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import ops
from torchinferno_b200.kernels.gemm import LinearWeight, linear
from torchinferno_b200.parts.base import (CacheSpec, LayerContext, Mixer, PartSpec, StateSpec, WeightSpec, build_part,
                                          register_part)

NO_WINDOW = 1 << 30        # what the kernel is told when every earlier token is visible


class KeptWindowAttention(Mixer):
    capturable = True       # (state is read and written by the kernel through the slots array)

    def __init__(self, *, hidden_size: int, heads: int, kv_heads: int, dim: int, scale: float, position: PartSpec | Mapping,
                 taps: int, window: int | None = None, keep_first: int = 0, row_norm_eps: float | None = None, sink: str | None = None,
                 gate: bool = False, q_name: str = "q", k_name: str = "k", o_name: str = "o", gate_name: str = "g",
                 sink_name: str = "sink", conv_suffix: str = ".conv", norm_suffix: str = ".norm",
                 dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if (window is not None and window < 1) or keep_first < 0 or taps < 1:
            raise ValueError("a window is positive, the kept tokens are not negative, and the convolution has at least one tap")
        if sink not in (None, "one", "learned"):
            raise ValueError(f"unknown sink {sink!r}; known: 'one', 'learned', None")
        self.hidden_size, self.heads, self.kv_heads, self.dim, self.scale = hidden_size, heads, kv_heads, dim, float(scale)
        self.taps, self.window, self.row_norm_eps = int(taps), None if window is None else int(window), row_norm_eps
        self.keep_first = 0 if window is None else int(keep_first)
        self.sink_kind, self.has_gate = sink, bool(gate)
        self.names = {"q": q_name, "k": k_name, "o": o_name, "g": gate_name, "sink": sink_name}
        self.conv_suffix, self.norm_suffix = conv_suffix, norm_suffix
        if not isinstance(position, PartSpec):
            position = PartSpec(**position)
        self.position = build_part("position", position, dtype=dtype, device=device)
        freq, _, interleaved = self.position.rotary_table()
        if freq.numel() and not interleaved or getattr(self.position, "amplitude", 1.0) != 1.0:
            raise ValueError("this attention's kernel turns the pairs (2i, 2i + 1) and takes no amplitude")

        def up(at: int) -> int:      # (every part of the product starts on a 16-byte boundary in bfloat16)
            return (at + 7) // 8 * 8
        self.k_off = up(heads * dim)
        self.g_off = up(self.k_off + kv_heads * dim)
        self.in_width = up(self.g_off + (heads * dim if gate else 0))
        self.in_weight: LinearWeight | None = None
        self.o_weight: LinearWeight | None = None
        self.q_conv = self.k_conv = self.q_norm_weight = self.k_norm_weight = self.sink = None

    def weight_specs(self) -> list[WeightSpec]:
        n, w = self.names, self.hidden_size
        std = w ** -0.5                     # (random weights: rows of about unit size from input of about unit size)
        specs = []
        for key, width in (("q", self.heads * self.dim), ("k", self.kv_heads * self.dim)):
            specs += [WeightSpec(n[key], (width, w), std=std),
                      WeightSpec(n[key] + self.conv_suffix, (width, self.taps), std=self.taps ** -0.5, role="vector")]
            if self.row_norm_eps is not None:
                specs.append(WeightSpec(n[key] + self.norm_suffix, (width,), init="about_one", std=0.1, role="vector"))
        if self.sink_kind == "learned":
            specs.append(WeightSpec(n["sink"], (self.heads,), std=1.0, role="vector"))
        if self.has_gate:
            specs.append(WeightSpec(n["g"], (self.heads * self.dim, w), std=std))
        specs.append(WeightSpec(n["o"], (w, self.heads * self.dim), std=(self.heads * self.dim) ** -0.5))
        return specs

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        first = weights[n["q"]]
        rows = torch.zeros((self.in_width, self.hidden_size), dtype=first.dtype, device=first.device)
        for key, at in (("q", 0), ("k", self.k_off), ("g", self.g_off)):
            if key != "g" or self.has_gate:
                part = weights[n[key]]
                rows[at:at + part.shape[0]] = part
        self.in_weight = LinearWeight(rows, few_rows_tcgen05=None)
        self.o_weight = LinearWeight(weights[n["o"]], few_rows_tcgen05=None)
        self.q_conv, self.k_conv = (weights[n[key] + self.conv_suffix].to(torch.float32).t().contiguous() for key in ("q", "k"))
        if self.row_norm_eps is not None:
            self.q_norm_weight, self.k_norm_weight = (weights[n[key] + self.norm_suffix].to(torch.float32).contiguous() for key in ("q", "k"))
        if self.sink_kind == "learned":
            self.sink = weights[n["sink"]].to(torch.float32).contiguous()
        elif self.sink_kind == "one":
            self.sink = torch.zeros(self.heads, dtype=torch.float32, device=first.device)

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(self.kv_heads, self.dim, self.window, keep_first=self.keep_first)

    def state_spec(self) -> StateSpec | None:
        floats = (self.taps - 1) * (self.heads + self.kv_heads) * self.dim
        return StateSpec((floats,), torch.float32) if floats else None

    def forward(self, x: torch.Tensor, ctx: LayerContext) -> torch.Tensor:
        kv, batch = ctx.kv, ctx.batch
        if kv is None or kv.keys is None or kv.values is None or not kv.writes:
            raise RuntimeError("this attention needs a cache binding with keys and values that it writes")
        if self.taps > 1 and ctx.state is None:
            raise RuntimeError("the convolution needs a state tensor")
        n, h, g, d = x.shape[0], self.heads, self.kv_heads, self.dim
        proj = linear(x, self.in_weight)                                    # [q | k | gate]
        q = torch.empty((n, h * d), dtype=x.dtype, device=x.device)
        ops.conv_norm_append(proj, 0, self.k_off, q, kv.keys, kv.values, self.q_conv, self.k_conv, batch.positions, kv.block_table,
                             batch.q_start, batch.slots, batch.n_entries, batch.max_q_len, h, g, d, freq=self.position.rotary_table()[0],
                             q_weight=self.q_norm_weight, k_weight=self.k_norm_weight, eps=self.row_norm_eps or 0.0,
                             state=ctx.state, error_word=ctx.error_word)
        out = torch.empty((n, h * d), dtype=x.dtype, device=x.device)
        ops.pooled_window_attention(
            q, out, batch.q_start, batch.kv_start, batch.slots, kv.keys, kv.values, kv.block_table, None, None, None, batch.n_entries,
            batch.max_q_len, h, g, window=self.window or NO_WINDOW, keep=self.keep_first, pool=0, scale=self.scale, sink=self.sink,
            gate=proj[:, self.g_off:self.g_off + h * d] if self.has_gate else None, error_word=ctx.error_word,
            max_kv_len=batch.max_kv_len)
        return linear(out, self.o_weight)


register_part("mixer", "kept_window_attention", KeptWindowAttention)
