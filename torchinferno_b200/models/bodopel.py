"""Bodopel as a description made of parts.

The embedding output is multiplied by a constant and a learned vector per position is added.  Every layer is a pre-norm block
with RMS norms whose gain is 1 + the stored weight; what a sublayer reads passes a short causal convolution that is added to it
(``causal_conv``).  The mixer is an attention inside a sliding window whose softmax weights are mixed across the heads
(``talking_heads_attention``: biases, queries and keys normed over all heads at once, a tanh cap on the scores, a bias that
falls with the logarithm of the distance, an element-wise output gate).  The feed-forward is W_down relu(W_up h)^2, or absent.
A range of layers may run several times with the same weights: each pass begins with the stage that adds the pass's vector, and
every run of a layer has a cache layer and carried rows of its own.  Tensor names: ``embed``, ``pos``, ``head``,
``final.norm``, ``loop.step``, and per layer ``l<i>.norm1`` / ``norm2``, ``l<i>.canon1`` / ``canon2``, ``l<i>.mix.*``,
``l<i>.mlp.*``.
"""
from __future__ import annotations

from torchinferno_b200.config.bodopel_config import BodopelConfig, BodopelLayer
from torchinferno_b200.config.registry import ArchitectureEntry, register_architecture
from torchinferno_b200.models.spec import BlockSpec, LayerCall, ModelSpec, StageCall
from torchinferno_b200.parts.base import PartSpec


def _mixer(layer: BodopelLayer, config: BodopelConfig) -> PartSpec:
    m = layer.mixer
    return PartSpec("talking_heads_attention", {
        "hidden_size": config.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "value_dim": m["vdim"],
        "scale": float(m["scale"]), "max_positions": config.max_positions, "window": layer.window, "softcap": layer.softcap,
        "bias": True, "row_norm_eps": config.eps, "distance_decay": True, "mix_heads": True, "gate": True}, prefix="mix.")


def _feed_forward(layer: BodopelLayer, config: BodopelConfig) -> PartSpec | None:
    if layer.mlp is None:
        return None
    return PartSpec("dense", {"hidden_size": config.width, "intermediate_size": layer.mlp["ff"], "activation": "relu2",
                              "up_name": "up", "down_name": "down"}, prefix="mlp.")


def build_bodopel(config: BodopelConfig) -> ModelSpec:
    def norm(name: str, prefix: str = "") -> PartSpec:
        return PartSpec("rmsnorm", {"width": config.width, "eps": config.eps, "weight_name": name, "weight_offset": 1.0}, prefix=prefix)

    def conv(name: str) -> PartSpec:
        return PartSpec("causal_conv", {"width": config.width, "taps": config.taps, "weight_name": name})

    blocks = []
    for i, layer in enumerate(config.layers):
        feed_forward = _feed_forward(layer, config)
        blocks.append(BlockSpec(PartSpec("prenorm", {
            "mixer": _mixer(layer, config), "mixer_norm": norm("norm1"), "mixer_input": conv("canon1"),
            "feed_forward": feed_forward, "feed_forward_norm": None if feed_forward is None else norm("norm2"),
            "feed_forward_input": None if feed_forward is None else conv("canon2")}), f"l{i}."))
    start, stop, times = config.loop if config.loop is not None else (0, 0, 0)
    stages = () if config.loop is None else (PartSpec("pass_vector", {"width": config.width, "passes": times}, prefix="loop."),)
    schedule: list[LayerCall | StageCall] = []
    caches = 0

    def run(layers: range) -> None:
        nonlocal caches
        for layer in layers:
            schedule.append(LayerCall(layer, caches))
            caches += 1

    run(range(start))
    for t in range(times):
        schedule.append(StageCall(0, t))
        run(range(start, stop))
    run(range(stop, len(config.layers)))
    return ModelSpec(
        architecture="Bodopel", hidden_size=config.width, vocab_size=config.vocab, max_positions=config.max_positions,
        embedding_name="embed", layers=tuple(blocks), schedule=tuple(schedule), final_norm=norm("norm", "final."),
        head_name="head", tie_head_to_embedding=False, config=config.to_dict(), stages=stages,
        embedding_scale=config.embedding_scale, position_embedding_name="pos")


BODOPEL = register_architecture(ArchitectureEntry(
    name="Bodopel", model_types=("bodopel",), config_class=BodopelConfig, build=build_bodopel))
