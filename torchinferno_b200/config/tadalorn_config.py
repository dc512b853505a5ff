"""Typed configuration of the Tadalorn design, read from a checkpoint's ``config.json``.

The file names the design under ``architecture``, gives the global sizes (``vocab``, ``width``), the norms' ``eps``, the factor of
every sublayer's way back into the residual (``residual_mult``), the cap on the logits (``logit_softcap``, 0 or null: none) and a
list ``layers`` whose entries each name a mixer ``type`` (``mlstm``, ``attention``, ``latent_attention``) with its sizes and
constants (``mixer``) and a feed-forward (``mlp``: dense or routed, or null).  An entry with ``weights_of`` runs with the tensors of
the layer it names.  No size or constant has a default: a missing key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from torchinferno_b200.config.model_config import ConfigError

MIXERS = ("mlstm", "attention", "latent_attention")
FEED_FORWARDS = ("dense", "moe")
# The design names no limit.  Positions are exact in the 32-bit floats the rotary angles are made from up to 2^24; the limit given
# here is what block tables and default pools are sized by when the user names none (EngineConfig.max_model_len).
MAX_POSITIONS = 1 << 20


def _need(data: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(data, Mapping) or key not in data:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return data[key]


def _integer(data: Mapping[str, Any], key: str, where: str, least: int) -> int:
    value = _need(data, key, where)
    if not isinstance(value, int) or isinstance(value, bool) or value < least:
        raise ConfigError(f"config.json: {where}.{key} must be an integer of at least {least}, got {value!r}")
    return value


def _positive(data: Mapping[str, Any], key: str, where: str) -> int:
    return _integer(data, key, where, 1)


def _number(data: Mapping[str, Any], key: str, where: str, positive: bool = True) -> float:
    value = _need(data, key, where)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or (positive and not float(value) > 0):
        raise ConfigError(f"config.json: {where}.{key} must be a {'positive ' if positive else ''}number, got {value!r}")
    return float(value)


def _rotary(mixer: Mapping[str, Any], at: str, width: int, exactly: bool) -> None:
    rot = _need(mixer, "rot", at)
    _number(rot, "base", at + ".rot")
    dims = _integer(rot, "dims", at + ".rot", 0)
    if dims % 2 or dims > width or (exactly and dims != width):
        raise ConfigError(f"config.json: {at}.rot.dims must be even and {'equal' if exactly else 'at most'} {width}, got {dims}")


@dataclass(frozen=True)
class TadalornLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None
    weights_of: int | None

    @property
    def window(self) -> int | None:
        mask = self.mixer.get("mask")
        return None if mask is None else mask["size"]

    @property
    def keep_first(self) -> int:
        mask = self.mixer.get("mask")
        return 0 if mask is None else mask["keep_first"]

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], index: int) -> "TadalornLayer":
        where = f"layers[{index}]"
        kind = _need(data, "type", where)
        if kind not in MIXERS:
            raise ConfigError(f"config.json: {where}.type={kind!r}; known mixers: {list(MIXERS)}")
        mixer = _need(data, "mixer", where)
        at = where + ".mixer"
        heads = _positive(mixer, "heads", at)
        _positive(mixer, "dim", at), _positive(mixer, "vdim", at)
        if kind == "mlstm":
            _number(mixer, "gate_cap", at)
        elif kind == "attention":
            if heads % _positive(mixer, "kv_heads", at):
                raise ConfigError(f"config.json: {at}.heads must be a multiple of kv_heads")
            if mixer["vdim"] != mixer["dim"]:
                raise ConfigError(f"config.json: {at}.vdim must equal dim (the values are the keys), got {mixer['vdim']} and {mixer['dim']}")
            _positive(mixer, "conv", at), _number(mixer, "scale", at, positive=False), _rotary(mixer, at, mixer["dim"], False)
            mask = _need(mixer, "mask", at)          # (null: every earlier token is visible)
            if mask is not None:
                _positive(mask, "size", at + ".mask"), _integer(mask, "keep_first", at + ".mask", 0)
        else:
            _positive(mixer, "rot_dim", at), _positive(mixer, "kv_rank", at), _number(mixer, "scale", at, positive=False)
            _rotary(mixer, at, mixer["rot_dim"], True)
        mlp = data.get("mlp")
        if mlp is not None:
            at = where + ".mlp"
            form = _need(mlp, "kind", at)
            if form not in FEED_FORWARDS:
                raise ConfigError(f"config.json: {at}.kind={form!r}; known: {list(FEED_FORWARDS)}")
            if form == "dense":
                _positive(mlp, "ff", at)
            else:
                router = _need(mlp, "router", at)
                if _positive(router, "top", at + ".router") > _positive(router, "experts", at + ".router"):
                    raise ConfigError(f"config.json: {at}.router.top exceeds the number of experts")
                _positive(_need(mlp, "expert", at), "ff", at + ".expert")
                if mlp.get("shared") is not None:
                    _positive(mlp["shared"], "ff", at + ".shared")
        source = data.get("weights_of")
        if source is not None:
            _integer(data, "weights_of", where, 0)
        return cls(kind, dict(mixer), None if mlp is None else dict(mlp), source)


@dataclass(frozen=True)
class TadalornConfig:
    vocab: int
    width: int
    layers: tuple[TadalornLayer, ...]
    eps: float
    residual_mult: float
    logit_softcap: float | None
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def source_of(self, index: int) -> int:
        """The layer whose tensors layer ``index`` runs with (itself, unless it names another)."""
        seen = {index}
        while self.layers[index].weights_of is not None:
            index = self.layers[index].weights_of
            if index in seen:
                raise ConfigError(f"config.json: layers[{index}].weights_of names itself in the end")
            seen.add(index)
        return index

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "TadalornConfig":
        where = "the model"
        layers = _need(data, "layers", where)
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a list with at least one entry")
        typed = tuple(TadalornLayer.from_dict(entry, i) for i, entry in enumerate(layers))
        for i, layer in enumerate(typed):
            j = layer.weights_of
            if j is None:
                continue
            if j >= len(typed):
                raise ConfigError(f"config.json: layers[{i}].weights_of={j}, but there are {len(typed)} layers")
            if (layer.type, layer.mixer, layer.mlp) != (typed[j].type, typed[j].mixer, typed[j].mlp):
                raise ConfigError(f"config.json: layers[{i}] names layer {j} in weights_of, but the rest of its entry differs from that layer's")
        cap = _need(data, "logit_softcap", where)
        if cap is not None and (isinstance(cap, bool) or not isinstance(cap, (int, float)) or cap < 0):
            raise ConfigError(f"config.json: logit_softcap must be a positive number (0 or null: none), got {cap!r}")
        config = cls(vocab=_positive(data, "vocab", where), width=_positive(data, "width", where), layers=typed,
                     eps=_number(_need(data, "norm", where), "eps", "norm"),
                     residual_mult=_number(data, "residual_mult", where, positive=False),
                     logit_softcap=float(cap) if cap else None, raw=dict(data))
        for i in range(len(typed)):
            config.source_of(i)
        return config

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)
