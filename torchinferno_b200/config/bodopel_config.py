"""Typed configuration of the Bodopel design, read from a checkpoint's ``config.json``.

The file names the design under ``architecture``, gives the global sizes (``vocab``, ``width``, ``max_positions``), the norms'
``eps``, the embedding's multiplier (``embedding.scale``), the taps of the input convolutions (``canon.taps``), optionally a
range of layers that runs several times (``loop.start`` / ``stop`` / ``times``) and a list ``layers`` whose entries each name a
mixer ``type`` (``attention``) with its sizes and constants (``mixer``) and a feed-forward (``mlp``, or null).  No size or
constant has a default: a missing key is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from torchinferno_b200.config.model_config import ConfigError

MIXERS = ("attention",)


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


@dataclass(frozen=True)
class BodopelLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None

    @property
    def window(self) -> int | None:
        mask = self.mixer["mask"]
        return None if mask is None else mask["size"]

    @property
    def softcap(self) -> float | None:
        return float(self.mixer["softcap"]) if self.mixer["softcap"] else None

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], index: int) -> "BodopelLayer":
        where = f"layers[{index}]"
        kind = _need(data, "type", where)
        if kind not in MIXERS:
            raise ConfigError(f"config.json: {where}.type={kind!r}; known mixers: {list(MIXERS)}")
        mixer = _need(data, "mixer", where)
        at = where + ".mixer"
        heads, kv_heads = _positive(mixer, "heads", at), _positive(mixer, "kv_heads", at)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {at}.heads must be a multiple of kv_heads")
        _positive(mixer, "dim", at), _positive(mixer, "vdim", at), _number(mixer, "scale", at)
        cap = _need(mixer, "softcap", at)
        if cap is not None and (isinstance(cap, bool) or not isinstance(cap, (int, float)) or cap < 0):
            raise ConfigError(f"config.json: {at}.softcap must be a positive number (0 or null: none), got {cap!r}")
        mask = _need(mixer, "mask", at)          # (null: every earlier token is visible)
        if mask is not None:
            _positive(mask, "size", at + ".mask")
        mlp = data.get("mlp")
        if mlp is not None:
            at = where + ".mlp"
            form = _need(mlp, "kind", at)
            if form != "dense":
                raise ConfigError(f"config.json: {at}.kind={form!r}; known: ['dense']")
            _positive(mlp, "ff", at)
        return cls(kind, dict(mixer), None if mlp is None else dict(mlp))


@dataclass(frozen=True)
class BodopelConfig:
    vocab: int
    width: int
    max_positions: int
    layers: tuple[BodopelLayer, ...]
    eps: float
    embedding_scale: float
    taps: int
    loop: tuple[int, int, int] | None          # (start, stop, times)
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "BodopelConfig":
        where = "the model"
        layers = _need(data, "layers", where)
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a list with at least one entry")
        typed = tuple(BodopelLayer.from_dict(entry, i) for i, entry in enumerate(layers))
        loop = None
        if data.get("loop") is not None:
            block = data["loop"]
            start, stop, times = _integer(block, "start", "loop", 0), _positive(block, "stop", "loop"), _positive(block, "times", "loop")
            if not start < stop <= len(typed):
                raise ConfigError(f"config.json: loop.start .. loop.stop = {start} .. {stop} is no range of the {len(typed)} layers")
            loop = (start, stop, times)
        return cls(vocab=_positive(data, "vocab", where), width=_positive(data, "width", where),
                   max_positions=_positive(data, "max_positions", where), layers=typed,
                   eps=_number(_need(data, "norm", where), "eps", "norm"),
                   embedding_scale=_number(_need(data, "embedding", where), "scale", "embedding", positive=False),
                   taps=_positive(_need(data, "canon", where), "taps", "canon"), loop=loop, raw=dict(data))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)
