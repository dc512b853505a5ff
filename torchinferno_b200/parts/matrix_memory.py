"""A matrix memory with exponential gates (the mLSTM of xLSTM), over state kept per request.

Per head, with q, k of ``dim`` and v of ``value_dim`` elements: q = W_q x * dim^(-1/2), k = W_k x, v = W_v x; a log input gate
i = cap tanh((w_i . x + b_i) / cap) and a log forget gate f = logsigmoid(cap tanh((w_f . x + b_f) / cap)) with ``gate_cap``;

    m_t = max(f + m_(t-1), i)                                                        (from 0 on)
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T,   n_t likewise with k alone
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)

Each head's o is divided by its root mean square (``eps``); the heads side by side are multiplied by a weight (``norm``) and by
sigmoid(W_g x), then projected by W_o.  S, n and m live in 32-bit in the cache manager's state slots (zero for a new request) and are
carried from step to step; the mixer keeps no keys.  q, k, v and the gate's logits are one product; the two gate rows per head are
summed in fp32 and stay fp32 in either mode (on long portions in bfloat16 by a product with fp32 output).  The kernels (csrc/matrix_memory.cu) take the step's whole ragged batch, prompt portions and
single tokens alike, and read it through its device arrays only.
"""
from __future__ import annotations

from typing import Mapping

import torch

from torchinferno_b200.kernels import ops
from torchinferno_b200.kernels.gemm import LinearWeight, linear
from torchinferno_b200.parts.base import LayerContext, Mixer, StateSpec, WeightSpec, register_part


MANY_ROWS = 128        # from this many rows on the gate rows are a library product


def up_to_eight(n: int) -> int:
    return (n + 7) // 8 * 8


class MatrixMemory(Mixer):
    capturable = True       # (state is read and written by the kernels through the slots array)

    def __init__(self, *, hidden_size: int, heads: int, dim: int, value_dim: int, gate_cap: float, eps: float = 1e-6,
                 q_name: str = "q", k_name: str = "k", v_name: str = "v", g_name: str = "g", o_name: str = "o", norm_name: str = "norm",
                 i_name: str = "i", f_name: str = "f", bias_suffix: str = ".b", dtype: torch.dtype, device: torch.device) -> None:
        super().__init__(dtype=dtype, device=device)
        if not gate_cap > 0:
            raise ValueError("the gates' cap is positive")
        self.hidden_size, self.heads, self.dim, self.value_dim = hidden_size, heads, dim, value_dim
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.names = {"q": q_name, "k": k_name, "v": v_name, "g": g_name, "o": o_name, "norm": norm_name, "i": i_name, "f": f_name,
                      "ib": i_name + bias_suffix, "fb": f_name + bias_suffix}
        # (every part of the product starts on a 16-byte boundary in bfloat16)
        self.k_off = up_to_eight(heads * dim)
        self.v_off = up_to_eight(self.k_off + heads * dim)
        self.g_off = up_to_eight(self.v_off + heads * value_dim)
        self.in_width = up_to_eight(self.g_off + heads * value_dim)
        self.in_weight: LinearWeight | None = None
        self.o_weight: LinearWeight | None = None
        self.gate_weight = self.gate_bias = self.norm_weight = self.gate_rows = None

    def weight_specs(self) -> list[WeightSpec]:
        n, w, qk, vv = self.names, self.hidden_size, self.heads * self.dim, self.heads * self.value_dim
        std = w ** -0.5                     # (random weights: rows of about unit size from input of about unit size)
        return [WeightSpec(n["q"], (qk, w), std=std), WeightSpec(n["k"], (qk, w), std=std), WeightSpec(n["v"], (vv, w), std=std),
                WeightSpec(n["g"], (vv, w), std=std), WeightSpec(n["o"], (w, vv), std=vv ** -0.5),
                WeightSpec(n["norm"], (vv,), init="about_one", std=0.1, role="vector"),
                WeightSpec(n["i"], (self.heads, w), std=std), WeightSpec(n["ib"], (self.heads,), std=1.0, role="vector"),
                WeightSpec(n["f"], (self.heads, w), std=std), WeightSpec(n["fb"], (self.heads,), init="about_one", std=1.0, role="vector")]

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        first = weights[n["q"]]
        rows = torch.zeros((self.in_width, self.hidden_size), dtype=first.dtype, device=first.device)
        for key, at in (("q", 0), ("k", self.k_off), ("v", self.v_off), ("g", self.g_off)):
            part = weights[n[key]]
            rows[at:at + part.shape[0]] = part
        self.in_weight = LinearWeight(rows, few_rows_tcgen05=None)
        self.o_weight = LinearWeight(weights[n["o"]], few_rows_tcgen05=None)
        if self.dtype == torch.bfloat16 and weights[n["i"]].dtype == weights[n["f"]].dtype == torch.bfloat16:
            rows = torch.zeros((up_to_eight(2 * self.heads), self.hidden_size), dtype=torch.bfloat16, device=first.device)
            rows[:self.heads], rows[self.heads:2 * self.heads] = weights[n["i"]], weights[n["f"]]
            self.gate_rows = LinearWeight(rows, few_rows_tcgen05=False)
        self.gate_weight = torch.cat([weights[n["i"]], weights[n["f"]]], dim=0).to(torch.float32).contiguous()
        self.gate_bias = torch.cat([weights[n["ib"]], weights[n["fb"]]], dim=0).to(torch.float32).contiguous()
        self.norm_weight = weights[n["norm"]].to(torch.float32).contiguous()
        if first.is_cuda and self.dim > ops.matrix_memory_max_dim():
            raise ValueError(f"heads with keys of {self.dim} do not fit the kernel (at most {ops.matrix_memory_max_dim()})")

    def state_spec(self) -> StateSpec:
        return StateSpec((ops.matrix_memory_state_floats(self.heads, self.dim, self.value_dim),), torch.float32)

    def forward(self, x: torch.Tensor, ctx: LayerContext) -> torch.Tensor:
        if ctx.state is None:
            raise RuntimeError("the matrix memory needs a state tensor")
        batch = ctx.batch
        proj = linear(x, self.in_weight)                                    # [q | k | v | gate]
        rows = torch.empty((x.shape[0], self.heads * self.value_dim), dtype=x.dtype, device=x.device)
        logits = None
        if self.gate_rows is not None and x.shape[0] >= MANY_ROWS and batch.max_q_len > 1:
            logits = linear(x, self.gate_rows, out_dtype=torch.float32)
        ops.matrix_memory(proj, 0, self.k_off, self.v_off, self.g_off, x, self.gate_weight, self.gate_bias, self.gate_cap, ctx.state,
                          batch.q_start, batch.slots, batch.n_entries, batch.max_q_len, self.norm_weight, self.eps, rows,
                          heads=self.heads, dim=self.dim, vdim=self.value_dim, q_scale=self.dim ** -0.5, logits=logits)
        return linear(rows, self.o_weight)


register_part("mixer", "matrix_memory", MatrixMemory)
