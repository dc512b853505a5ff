"""A plain, slow Bodopel forward pass for the tests: whole sequences, no cache, one function per mechanism.

Bodopel is a decoder-only design of pre-norm layers with learned absolute positions.  What a sublayer reads passes a short
causal convolution per channel that is added to it; the mixer is a grouped attention inside a sliding window whose
queries and keys are normed over all heads at once, whose scores pass a tanh cap and lose a logarithm of the distance,
whose softmax weights are mixed across the heads, and whose output is gated; the feed-forward is a squared relu between
two products.  A range of layers may run several times, each pass opened by a vector of its own.  This file shares no code
with ``torchinferno_b200``: it reads config.json and model.safetensors itself and computes on the CPU in float64, so that
its own rounding does not count against the engine.

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
def rms_norm(x, gain, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * gain


def zero_centred_norm(x, stored, eps):
    """The gain is 1 + stored."""
    return rms_norm(x, 1 + stored, eps)


def input_convolution(h, taps_of):
    """h_t + sum_j taps_of[:, j] * h_(t - taps + 1 + j), channel by channel; rows before the first are zero."""
    taps = taps_of.shape[1]
    out = h.clone()
    for t in range(h.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += taps_of[:, j] * h[s]
    return out


# ---------------------------------------------------------------- attention
def capped(scores, cap):
    return cap * torch.tanh(scores / cap) if cap else scores


def distance_loss(r1, r2, distance):
    """What head h's score loses at each distance: r1[h] * ln(1 + r2[h] * distance); [H, *distance.shape]."""
    shape = (-1,) + (1,) * distance.dim()
    return r1.view(shape) * torch.log(1 + r2.view(shape) * distance.to(F))


def window_weights(scores, window):
    """Softmax over the keys j of row i with 0 <= i - j < window; scores [H, T, T]."""
    T = scores.shape[-1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & (i - j < window)
    return torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)


def mix_heads(weights, talk):
    """weight_h(i, j) <- sum_g talk[h, g] weight_g(i, j)."""
    return torch.einsum("hg,gij->hij", talk, weights)


def attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.norm"], eps).view(T, H, d)       # (normed over all heads at once)
    k = rms_norm(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.norm"], eps).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    kh, vh = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    scores = capped(torch.einsum("ihd,jhd->hij", q, kh) * m["scale"], m["softcap"])
    distance = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    scores = scores - distance_loss(w[p + "r1"], w[p + "r2"], distance)
    window = T if m["mask"] is None else m["mask"]["size"]
    weights = mix_heads(window_weights(scores, window), w[p + "talk"])
    rows = torch.einsum("hij,jhd->ihd", weights, vh).reshape(T, H * dv)
    return (rows * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------ feed-forward
def squared_relu_unit(h, w, p):
    return torch.relu(h @ w[p + "up"].T).pow(2) @ w[p + "down"].T


# -------------------------------------------------------------------- model
def layer_runs(config):
    """(layer, pass whose vector is added ahead of it, or None) in the order of execution."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(start)]
    for t in range(loop["times"]):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


def forward(config, w, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from its first token (and the residual stream after every layer run)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = w["embed"][tokens] * config["embedding"]["scale"] + w["pos"][:tokens.numel()]
    after = []
    for i, opens in layer_runs(config):
        p, layer = f"l{i}.", config["layers"][i]
        if opens is not None:
            x = x + w["loop.step"][opens]
        h = input_convolution(zero_centred_norm(x, w[p + "norm1"], eps), w[p + "canon1"])
        x = x + attention(h, w, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = input_convolution(zero_centred_norm(x, w[p + "norm2"], eps), w[p + "canon2"])
            x = x + squared_relu_unit(h, w, p + "mlp.")
        after.append(x)
    logits = zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if return_layers else logits
