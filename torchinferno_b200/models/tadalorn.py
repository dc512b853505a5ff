"""Tadalorn as a description made of parts.

Every layer is a ``postnorm`` block: its sublayers read the residual stream as it is, and what they leave is RMS-normed and added
with one constant factor.  The mixer is a matrix memory with exponential gates (``matrix_memory``, the mLSTM of xLSTM), a grouped
attention inside a sliding window that keeps the first tokens in sight (``kept_window_attention``: a short convolution on queries and
keys, values that are the convolved keys, a norm over all heads at once, rotary on part of a head, one added to the softmax's
denominator, an output gate) or an attention over a low-rank latent (``latent_attention``: a learned number per head in the
denominator, an output gate).  The feed-forward is a gated unit with SiLU (``swiglu``), experts with the erf form of gelu behind a
router with a bias (``routed_experts``, a softmax over the chosen logits, a shared expert), or absent.  A layer may run with another
layer's tensors, with a cache or state of its own.  Logits pass c * tanh(. / c).  Tensor names: ``embed``, ``head``,
``final.norm``, and per layer ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from torchinferno_b200.config.registry import ArchitectureEntry, register_architecture
from torchinferno_b200.config.tadalorn_config import MAX_POSITIONS, TadalornConfig, TadalornLayer
from torchinferno_b200.models.spec import BlockSpec, LayerCall, ModelSpec
from torchinferno_b200.parts.base import PartSpec


def _mixer(layer: TadalornLayer, config: TadalornConfig) -> PartSpec:
    m = layer.mixer
    if layer.type == "mlstm":
        return PartSpec("matrix_memory", {
            "hidden_size": config.width, "heads": m["heads"], "dim": m["dim"], "value_dim": m["vdim"],
            "gate_cap": float(m["gate_cap"]), "eps": config.eps}, prefix="mix.")
    if layer.type == "attention":
        position = PartSpec("rotary", {"head_dim": m["dim"], "theta": float(m["rot"]["base"]), "rot_dim": m["rot"]["dims"],
                                       "interleaved": True, "exact": True})
        return PartSpec("kept_window_attention", {
            "hidden_size": config.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "scale": float(m["scale"]),
            "position": position, "taps": m["conv"], "window": layer.window, "keep_first": layer.keep_first,
            "row_norm_eps": config.eps, "sink": "one", "gate": True}, prefix="mix.")
    return PartSpec("latent_attention", {
        "hidden_size": config.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
        "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "rot_base": float(m["rot"]["base"]), "rot_dims": m["rot"]["dims"],
        "eps": config.eps, "sink": True, "gate": True}, prefix="mix.")


def _feed_forward(layer: TadalornLayer, config: TadalornConfig) -> PartSpec | None:
    mlp = layer.mlp
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", {"hidden_size": config.width, "intermediate_size": mlp["ff"], "gate_name": "gate",
                                   "up_name": "up", "down_name": "down"}, prefix="mlp.")
    shared = mlp.get("shared")
    # (softmax scores divided by the sum of the chosen ones are the softmax over the chosen logits)
    return PartSpec("routed_experts", {
        "hidden_size": config.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "expert_size": mlp["expert"]["ff"], "activation": "gelu", "scores": "softmax", "normalize": True, "router_bias": True,
        "shared_size": 0 if shared is None else shared["ff"]}, prefix="mlp.")


def build_tadalorn(config: TadalornConfig) -> ModelSpec:
    def norm(name: str, prefix: str = "") -> PartSpec:
        return PartSpec("rmsnorm", {"width": config.width, "eps": config.eps, "weight_name": name}, prefix=prefix)

    blocks: list[BlockSpec] = []
    block_of: dict[int, int] = {}          # layer that owns tensors -> its block
    for i, layer in enumerate(config.layers):
        if layer.weights_of is not None:
            continue
        feed_forward = _feed_forward(layer, config)
        block_of[i] = len(blocks)
        blocks.append(BlockSpec(PartSpec("postnorm", {
            "mixer": _mixer(layer, config), "mixer_norm": norm("norm1"), "feed_forward": feed_forward,
            "feed_forward_norm": None if feed_forward is None else norm("norm2"), "residual_scale": config.residual_mult}), f"l{i}."))
    schedule, caches = [], 0
    for i, layer in enumerate(config.layers):
        cached = layer.type != "mlstm"
        schedule.append(LayerCall(block_of[config.source_of(i)], caches if cached else None))
        caches += cached
    return ModelSpec(
        architecture="Tadalorn", hidden_size=config.width, vocab_size=config.vocab, max_positions=MAX_POSITIONS,
        embedding_name="embed", layers=tuple(blocks), schedule=tuple(schedule), final_norm=norm("norm", "final."),
        head_name="head", tie_head_to_embedding=False, config=config.to_dict(), logit_softcap=config.logit_softcap)


TADALORN = register_architecture(ArchitectureEntry(
    name="Tadalorn", model_types=("tadalorn",), config_class=TadalornConfig, build=build_tadalorn))
