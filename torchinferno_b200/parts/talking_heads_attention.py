"""Grouped attention inside a sliding window whose softmax weights are mixed across the heads before they meet the values.

q = W_q x, k = W_k x, v = W_v x (with biases when ``bias``); with ``row_norm_eps`` the whole q row and the whole k row, all
heads at once, are divided by their root mean square and multiplied by a weight per element (``q.norm`` / ``k.norm``,
multiplied in as stored).  There is no rotation: positions enter through the window (a query at i sees j with 0 <= i - j <
``window``; None: every earlier token) and, with ``distance_decay``, through a bias per head that falls with the logarithm of
the distance:

    s_h(i, j) = cap(q_i . k_j * scale) - r1[h] * ln(1 + r2[h] * (i - j)),      cap(s) = softcap * tanh(s / softcap) (None: s)
    w_h(i, .) = softmax over the visible j;      m_h(i, j) = sum_g talk[h, g] w_g(i, j)      (``mix_heads``; else m = w)

Head h applies m_h to the values of key/value head h // (heads / kv_heads); the heads side by side are multiplied element by
element by sigmoid(W_g x) (``gate``) and projected by W_o.

When the model is bound the bias is laid out by distance, [heads, span] with span the window (or the model's last position),
so no kernel takes a logarithm.  All input projections are one product; the kernels are in csrc/talking_heads.cu.
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import ops
from torchinferno_b200.kernels.gemm import LinearWeight, linear
from torchinferno_b200.parts.base import CacheSpec, LayerContext, Mixer, WeightSpec, register_part

NO_WINDOW = 1 << 30        # what the kernels are told when every earlier token is visible


class TalkingHeadsAttention(Mixer):
    capturable = True

    def __init__(self, *, hidden_size: int, heads: int, kv_heads: int, dim: int, value_dim: int, scale: float,
                 max_positions: int, window: int | None = None, softcap: float | None = None, bias: bool = False,
                 row_norm_eps: float | None = None, distance_decay: bool = False, mix_heads: bool = True, gate: bool = False,
                 q_name: str = "q", k_name: str = "k", v_name: str = "v", o_name: str = "o", gate_name: str = "g",
                 talk_name: str = "talk", decay_names: tuple[str, str] = ("r1", "r2"), bias_suffix: str = ".b",
                 norm_suffix: str = ".norm", dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if window is not None and window < 1:
            raise ValueError("a window is positive")
        if softcap is not None and not softcap > 0:
            raise ValueError("a cap is positive")
        self.hidden_size, self.heads, self.kv_heads, self.dim, self.value_dim = hidden_size, heads, kv_heads, dim, value_dim
        self.scale, self.softcap, self.row_norm_eps = float(scale), softcap, row_norm_eps
        self.window = None if window is None else int(window)
        self.span = max_positions if window is None else min(int(window), max_positions)      # distances that can be seen
        self.has_bias, self.has_decay, self.has_mix, self.has_gate = bool(bias), bool(distance_decay), bool(mix_heads), bool(gate)
        self.names = {"q": q_name, "k": k_name, "v": v_name, "o": o_name, "g": gate_name, "talk": talk_name,
                      "r1": decay_names[0], "r2": decay_names[1]}
        self.bias_suffix, self.norm_suffix = bias_suffix, norm_suffix
        qw, kw, vw = heads * dim, kv_heads * dim, kv_heads * value_dim

        def up(at: int) -> int:      # (every part of the product starts on a 16-byte boundary in bfloat16)
            return (at + 7) // 8 * 8
        self.k_off = up(qw)
        self.v_off = up(self.k_off + kw)
        self.g_off = up(self.v_off + vw)
        self.in_width = up(self.g_off + (heads * value_dim if gate else 0))
        self.in_weight: LinearWeight | None = None
        self.o_weight: LinearWeight | None = None
        self.q_bias = self.k_bias = self.v_bias = self.q_norm_weight = self.k_norm_weight = None
        self.bias_by_distance = self.talk = self.talk_hi = self.talk_lo = None

    def weight_specs(self) -> list[WeightSpec]:
        n, w = self.names, self.hidden_size
        std = w ** -0.5                     # (random weights: rows of about unit size from normed input)
        widths = {"q": self.heads * self.dim, "k": self.kv_heads * self.dim, "v": self.kv_heads * self.value_dim}
        specs = []
        for key, width in widths.items():
            specs.append(WeightSpec(n[key], (width, w), std=std))
            if self.has_bias:
                specs.append(WeightSpec(n[key] + self.bias_suffix, (width,), std=0.5, role="vector"))
            if self.row_norm_eps is not None and key != "v":
                specs.append(WeightSpec(n[key] + self.norm_suffix, (width,), init="about_one", std=0.1, role="vector"))
        if self.has_decay:
            # (random weights: positive numbers of about one half and one quarter of a unit)
            specs += [WeightSpec(n["r1"], (self.heads,), init="about_one", std=0.3, role="vector"),
                      WeightSpec(n["r2"], (self.heads,), init="about_one", std=0.2, role="vector")]
        if self.has_mix:
            specs.append(WeightSpec(n["talk"], (self.heads, self.heads), init="about_identity", std=0.3, role="vector"))
        if self.has_gate:
            specs.append(WeightSpec(n["g"], (self.heads * self.value_dim, w), std=std))
        specs.append(WeightSpec(n["o"], (w, self.heads * self.value_dim), std=(self.heads * self.value_dim) ** -0.5))
        return specs

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        first = weights[n["q"]]
        rows = torch.zeros((self.in_width, self.hidden_size), dtype=first.dtype, device=first.device)
        for key, at in (("q", 0), ("k", self.k_off), ("v", self.v_off), ("g", self.g_off)):
            if key != "g" or self.has_gate:
                part = weights[n[key]]
                rows[at:at + part.shape[0]] = part
        self.in_weight = LinearWeight(rows, few_rows_tcgen05=None)
        self.o_weight = LinearWeight(weights[n["o"]], few_rows_tcgen05=None)

        def vector(name):
            return weights[name].to(torch.float32).contiguous()

        if self.has_bias:
            self.q_bias, self.k_bias, self.v_bias = (vector(n[key] + self.bias_suffix) for key in ("q", "k", "v"))
        if self.row_norm_eps is not None:
            self.q_norm_weight, self.k_norm_weight = (vector(n[key] + self.norm_suffix) for key in ("q", "k"))
        if self.has_decay:
            r1, r2 = vector(n["r1"]).double(), vector(n["r2"]).double()
            distance = torch.arange(self.span, dtype=torch.float64, device=r1.device)
            self.bias_by_distance = (-r1[:, None] * torch.log1p(r2[:, None] * distance[None, :])).to(torch.float32).contiguous()
        self.talk = vector(n["talk"]) if self.has_mix else torch.eye(self.heads, dtype=torch.float32, device=first.device)
        if self.dtype == torch.bfloat16 and self.heads <= 64:
            padded = 16 if self.heads <= 16 else 32 if self.heads <= 32 else 64
            wide = torch.zeros((padded, padded), dtype=torch.float32, device=first.device)
            wide[:self.heads, :self.heads] = self.talk
            self.talk_hi = wide.to(torch.bfloat16)
            rest = (wide - self.talk_hi.float()).to(torch.bfloat16)
            self.talk_lo = rest if bool(rest.abs().max() > 0) else None      # (read once, when the model is bound)

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(self.kv_heads, self.dim, self.window, None if self.value_dim == self.dim else self.value_dim)

    def forward(self, x: torch.Tensor, ctx: LayerContext) -> torch.Tensor:
        kv, batch = ctx.kv, ctx.batch
        if kv is None or kv.keys is None or kv.values is None or not kv.writes:
            raise RuntimeError("this attention needs a cache binding with keys and values that it writes")
        n, h, g = x.shape[0], self.heads, self.kv_heads
        proj = linear(x, self.in_weight)                                    # [q | k | v | gate]
        q = torch.empty((n, h * self.dim), dtype=x.dtype, device=x.device)
        ops.row_norm_append(proj, 0, self.k_off, self.v_off, q, kv.keys, kv.values, batch.positions, batch.token_slot, kv.block_table,
                            h, g, self.dim, self.value_dim, eps=self.row_norm_eps or 0.0, q_bias=self.q_bias, k_bias=self.k_bias,
                            v_bias=self.v_bias, q_weight=self.q_norm_weight, k_weight=self.k_norm_weight, error_word=ctx.error_word)
        out = torch.empty((n, h * self.value_dim), dtype=x.dtype, device=x.device)
        ops.talking_heads_attention(
            q, out, batch.q_start, batch.kv_start, batch.slots, batch.positions, kv.keys, kv.values, kv.block_table, batch.n_entries,
            batch.max_q_len, h, g, window=self.window or NO_WINDOW, scale=self.scale, softcap=self.softcap or 0.0,
            bias=self.bias_by_distance, talk=self.talk, talk_hi=self.talk_hi, talk_lo=self.talk_lo,
            gate=proj[:, self.g_off:self.g_off + h * self.value_dim] if self.has_gate else None, max_kv_len=batch.max_kv_len,
            error_word=ctx.error_word)
        return linear(out, self.o_weight)


register_part("mixer", "talking_heads_attention", TalkingHeadsAttention)
