"""A plain, slow Tadalorn forward pass for the tests: whole sequences, no cache, one function per mechanism.

Tadalorn is a decoder-only design whose sublayers read the residual stream as it is and are normed on their way back into it.
Its mixers are a matrix memory with exponential gates (xLSTM's mLSTM), a grouped attention inside a sliding window that keeps
the first tokens in sight and whose values are its keys ahead of norm and rotation, and an attention over a low-rank latent;
its feed-forwards are a gated unit, routed experts beside a shared one, or absent.  A layer may run with another layer's
tensors.  This file shares no code with ``torchinferno_b200``: it reads config.json and model.safetensors itself and computes on
the CPU in float64, token by token where the design is a recurrence, so that its own rounding does not count against the engine.

Notation: T tokens, W the model width, x the residual stream [T, W]; w the checkpoint's tensors by name.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

F = torch.float64


def read_model_folder(folder, dtype=F):
    from safetensors import safe_open
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    weights = {}
    with safe_open(str(folder / "model.safetensors"), framework="pt", device="cpu") as handle:
        for name in handle.keys():
            t = handle.get_tensor(name)
            weights[name] = t.to(dtype) if t.is_floating_point() else t
    return config, weights


# ------------------------------------------------------------- small pieces
def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu(z):
    """z times the normal distribution's cumulative function at z."""
    return z * 0.5 * (1 + torch.erf(z / math.sqrt(2)))


def rotate_pairs(x, positions, base, dims):
    """Rotary on the first ``dims`` elements of the last axis of x [T, ..., d]; element 2i pairs with 2i + 1,
    angle = position * base^(-2i / dims); the rest pass unchanged."""
    i = torch.arange(dims // 2, dtype=F)
    angle = positions.to(F)[:, None] * (torch.tensor(float(base), dtype=F) ** (-2 * i / dims))[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = angle.cos().reshape(shape), angle.sin().reshape(shape)
    even, odd = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = even * cos - odd * sin
    out[..., 1:dims:2] = odd * cos + even * sin
    return out


def channel_convolution(u, taps_of):
    """y_t = sum_j taps_of[:, j] * u_(t - taps + 1 + j), channel by channel; rows before the first are zero."""
    taps = taps_of.shape[1]
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += taps_of[:, j] * u[s]
    return out


# ------------------------------------------------------------------- mixers
def seen_keys(T, window, first):
    """[T, T] bool: row i sees column j.  ``window`` None: every earlier token."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    causal = j <= i
    return causal if window is None else causal & ((i - j < window) | (j < first))


def softmax_with_sink(scores, seen, sink):
    """exp(s_j) / (exp(sink) + sum over the seen j of exp(s_j)); scores [H, T, T], sink [H]."""
    s = scores.masked_fill(~seen, -math.inf)
    with_sink = torch.cat([s, sink.view(-1, 1, 1).expand(-1, s.shape[1], 1)], dim=-1)
    return torch.softmax(with_sink, dim=-1)[..., :-1]


def window_attention(h, w, p, m, eps, positions):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = channel_convolution(h @ w[p + "q"].T, w[p + "q.conv"])
    k = channel_convolution(h @ w[p + "k"].T, w[p + "k.conv"])
    v = k.view(T, G, d)                                                          # (ahead of norm and rotation)
    q = rms_norm(q, w[p + "q.norm"], eps).view(T, H, d)                          # (normed over all heads at once)
    k = rms_norm(k, w[p + "k.norm"], eps).view(T, G, d)
    q, k = (rotate_pairs(part, positions, m["rot"]["base"], m["rot"]["dims"]) for part in (q, k))
    kh, vh = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, kh) * m["scale"]
    mask = m.get("mask")
    seen = seen_keys(T, None if mask is None else mask["size"], 0 if mask is None else mask["keep_first"])
    weights = softmax_with_sink(scores, seen, torch.zeros(H, dtype=h.dtype))     # (one added to the denominator)
    rows = torch.einsum("hij,jhd->ihd", weights, vh).reshape(T, H * d)
    return (rows * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps, positions):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    q_plain, q_rot = q[..., :D], rotate_pairs(q[..., D:].contiguous(), positions, base, dims)
    dkv = h @ w[p + "dkv"].T
    latent = rms_norm(dkv[:, :C], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(dkv[:, C:].contiguous(), positions, base, dims)         # [T, R], one for all heads
    k_plain = (latent @ w[p + "uk"].T).view(T, H, D)
    value = (latent @ w[p + "uv"].T).view(T, H, V)
    scores = (torch.einsum("thd,shd->hts", q_plain, k_plain) + torch.einsum("thr,sr->hts", q_rot, k_rot)) * m["scale"]
    weights = softmax_with_sink(scores, seen_keys(T, None, 0), w[p + "sink"])
    rows = torch.einsum("hts,shv->thv", weights, value).reshape(T, H * V)
    return (rows * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def memory_gates(h, w, p, cap):
    """(log input gate, log forget gate), [T, heads] each."""
    def capped(name):
        return cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    return capped("i"), -torch.log1p(torch.exp(-capped("f")))


def matrix_memory(q, k, v, log_in, log_forget):
    """The recurrence of one sequence, token by token: q, k [T, H, D], v [T, H, V], gates [T, H]; returns [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    top = torch.zeros(H, dtype=q.dtype)
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        new_top = torch.maximum(log_forget[t] + top, log_in[t])
        keep, take = torch.exp(log_forget[t] + top - new_top), torch.exp(log_in[t] - new_top)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        top = new_top
        bottom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / bottom[:, None]
    return out


def mlstm(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    o = matrix_memory(q, k, v, *memory_gates(h, w, p, m["gate_cap"]))
    rows = unit_rms(o, eps).reshape(T, H * V) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return rows @ w[p + "o"].T


# ------------------------------------------------------------ feed-forwards
def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def gelu_expert(h, up, down):
    return gelu(h @ up.T) @ down.T


def routed_experts(h, w, p, mlp, gaps=None):
    """The ``top`` largest logits (with the router's bias) are chosen, lowest index first among equals; the weights are a
    softmax over the chosen ones.  ``gaps`` (a list per token) collects how far the last chosen logit lies above the first one
    left out."""
    experts, top = mlp["router"]["experts"], mlp["router"]["top"]
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ranked = sorted(range(experts), key=lambda e: (-float(z[t, e]), e))
        chosen = ranked[:top]
        if gaps is not None and top < experts:
            gaps[t].append(float(z[t, ranked[top - 1]] - z[t, ranked[top]]))
        weights = torch.softmax(z[t, chosen], dim=0)
        for weight, e in zip(weights, chosen):
            out[t] += weight * gelu_expert(h[t], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    if mlp.get("shared"):
        out = out + gelu_expert(h, w[p + "shared.up"], w[p + "shared.down"])
    return out


# -------------------------------------------------------------------- model
def tensors_of(config, i):
    """The layer whose tensors layer i runs with."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config, w, tokens, return_layers=False, gaps=None):
    """Logits [T, vocab] of one sequence from its first token (and the residual stream after every layer).  ``gaps``: a list of
    one list per token, filled with the routers' margins at that token."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(tokens))
    eps, back = config["norm"]["eps"], config["residual_mult"]
    x, after = w["embed"][tokens], []
    for i in range(len(config["layers"])):
        j = tensors_of(config, i)
        layer, p = config["layers"][j], f"l{j}."
        m = layer["mixer"]
        if layer["type"] == "attention":
            y = window_attention(x, w, p + "mix.", m, eps, positions)
        elif layer["type"] == "latent_attention":
            y = latent_attention(x, w, p + "mix.", m, eps, positions)
        elif layer["type"] == "mlstm":
            y = mlstm(x, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + back * rms_norm(y, w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = gated_unit(x, w, p + "mlp.") if mlp["kind"] == "dense" else routed_experts(x, w, p + "mlp.", mlp, gaps)
            x = x + back * rms_norm(y, w[p + "norm2"], eps)
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = config["logit_softcap"]
    logits = cap * torch.tanh(logits / cap) if cap else logits
    return (logits, torch.stack(after)) if return_layers else logits
