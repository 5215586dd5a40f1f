"""Relulix configuration: the keys of its config.json.

A small decoder-only family that lists its layers one by one and mixes windowed attention with retention::

    architecture   "Relulix"
    vocab, width
    embedding      {"scale"}         the looked-up row is multiplied by it
    layers         [{"type": "attention" | "retention", "mixer": {...}, "mlp": {...} | null}, ...]
    norm           {"eps"}

``mixer`` of an ``attention`` layer: heads, kv_heads, dim, vdim, scale, softcap (absent or 0: no cap), mask {size}
(the newest keys a token sees, its own included; absent: all), rot {base, dims, scaling {factor, original, fast, slow}
| absent}, kv_from (absent, or the number of an earlier attention layer whose keys and values this one reads; that
layer must have keys and values of its own, with as many heads of the same sizes and the same rotation).
``mixer`` of a ``retention`` layer: heads, dim, vdim, decay (one number per head), rot.
``mlp``: kind "moe" {expert {ff, limit}, router {experts, top}}.

No size has a default: a key that the model needs and config.json lacks is an error.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Optional

from .base import ConfigError, ModelConfig

LAYER_TYPES = ("attention", "retention")
WHO = "RelulixConfig"


def _need(d: Any, key: str, where: str, kind=(int, float)):
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"{WHO}: {where} lacks '{key}'")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, kind):
        raise ConfigError(f"{WHO}: {where}.{key} has the wrong type: {v!r}")
    return v


def _positive(d: Any, keys, where: str) -> None:
    for k in keys:
        if _need(d, k, where, int) <= 0:
            raise ConfigError(f"{WHO}: {where}.{k} must be positive")


def _check_rot(rot: Any, dim: int, where: str) -> None:
    dims = _need(rot, "dims", where, int)
    if dims <= 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{WHO}: {where}.dims must be even, positive and at most the head's dim")
    if not _need(rot, "base", where) > 1:
        raise ConfigError(f"{WHO}: {where}.base must be beyond 1")
    if rot.get("scaling") is not None:
        for k in ("factor", "original", "fast", "slow"):
            if not _need(rot["scaling"], k, where + ".scaling") > 0:
                raise ConfigError(f"{WHO}: {where}.scaling.{k} must be positive")


def _check_attention(m: Any, where: str) -> None:
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{WHO}: {where}.heads must be a multiple of kv_heads")
    if not _need(m, "scale", where) > 0:
        raise ConfigError(f"{WHO}: {where}.scale must be positive")
    if m.get("softcap") is not None and _need(m, "softcap", where) < 0:
        raise ConfigError(f"{WHO}: {where}.softcap cannot be negative")
    if m.get("mask") is not None:
        _positive(m["mask"], ("size",), where + ".mask")
    _check_rot(m.get("rot"), m["dim"], where + ".rot")


def _check_retention(m: Any, where: str) -> None:
    _positive(m, ("heads", "dim", "vdim"), where)
    decay = m.get("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != m["heads"]:
        raise ConfigError(f"{WHO}: {where}.decay must list one number per head")
    for d in decay:
        if isinstance(d, bool) or not isinstance(d, (int, float)) or not 0 <= d <= 1:
            raise ConfigError(f"{WHO}: {where}.decay holds {d!r}; every decay lies between 0 and 1")
    _check_rot(m.get("rot"), m["dim"], where + ".rot")


def _check_kv_from(layers, i: int, where: str) -> None:
    m = layers[i]["mixer"]
    j = m.get("kv_from")
    if j is None:
        return
    j = _need(m, "kv_from", where, int)
    if not 0 <= j < i or layers[j]["type"] != "attention" or layers[j]["mixer"].get("kv_from") is not None:
        raise ConfigError(f"{WHO}: {where}.kv_from is {j}; it must name an earlier attention layer that has keys and "
                          f"values of its own")
    src = layers[j]["mixer"]
    for k in ("kv_heads", "dim", "vdim", "rot"):
        if src[k] != m[k]:
            raise ConfigError(f"{WHO}: {where}.{k} differs from that of layer {j}, whose keys and values it reads")


def _check_mlp(mlp: Any, where: str) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"{WHO}: {where}.kind must be 'moe'")
    _positive(mlp.get("expert"), ("ff",), where + ".expert")
    if not _need(mlp["expert"], "limit", where + ".expert") > 0:
        raise ConfigError(f"{WHO}: {where}.expert.limit must be positive")
    router = mlp.get("router")
    _positive(router, ("experts", "top"), where + ".router")
    if router["top"] > router["experts"]:
        raise ConfigError(f"{WHO}: {where}.router.top exceeds the number of experts")


@dataclasses.dataclass
class RelulixConfig(ModelConfig):
    architecture: ClassVar[str] = "Relulix"
    model_types: ClassVar[tuple[str, ...]] = ("relulix",)

    vocab: int = 0
    width: int = 0
    layers: tuple = ()
    norm: Optional[dict] = None
    embedding: Optional[dict] = None

    def to_dict(self) -> dict[str, Any]:
        out = super().to_dict()
        out["architecture"] = self.architecture
        out["layers"] = list(self.layers)
        return out

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError(f"{WHO}: vocab and width must be positive")
        if not self.layers:
            raise ConfigError(f"{WHO}: 'layers' is empty")
        if not _need(self.norm, "eps", "norm") > 0:
            raise ConfigError(f"{WHO}: norm.eps must be positive")
        _need(self.embedding, "scale", "embedding")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, dict) else layer
            if kind not in LAYER_TYPES:
                raise ConfigError(f"{WHO}: {where}.type is {kind!r}; known: {LAYER_TYPES}")
            if kind == "attention":
                _check_attention(layer.get("mixer"), where + ".mixer")
                _check_kv_from(self.layers, i, where + ".mixer")
            else:
                _check_retention(layer.get("mixer"), where + ".mixer")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], where + ".mlp")

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def embedding_scale(self) -> float:
        return float(self.embedding["scale"])
