"""Papusun configuration: the keys of its config.json.

A small decoder-only family that lists its layers one by one::

    architecture   "Papusun"
    vocab, width
    layers         [{"type": "parallel" | "latent_attention", "mixer": {...}, "mlp": {...} | null}, ...]
    norm           {"eps"}
    token_side     {"dim"}           numbers per layer of every token's own row
    logit_scale                      multiplies the logits

``mixer`` of a ``parallel`` layer: left {heads, kv_heads, dim, vdim, scale, softcap (absent or 0: no cap), rot {base,
dims, scaling {factor, low, high, original} | absent}}, right {heads, kv_heads, dim, vdim, conv (taps)}, left_scale,
right_scale: attention and a gated delta rule side by side.
``mixer`` of a ``latent_attention`` layer: heads, dim (unrotated query/key size per head), rot_dim (rotated), vdim,
q_rank, kv_rank, scale, mask {size} (the newest keys a token sees, its own included; absent: all), rot {base, dims},
kv_from (absent, or the number of an earlier latent layer whose latents and rotated key parts this one reads; that layer
must have its own, of the same sizes and with the same rotation).
``mlp``: kind "dense" {ff}.

No size has a default: a key that the model needs and config.json lacks is an error.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Optional

from .base import ConfigError, ModelConfig

LAYER_TYPES = ("parallel", "latent_attention")
WHO = "PapusunConfig"


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


def _check_rot(rot: Any, dim: int, where: str, scaled: bool) -> None:
    dims = _need(rot, "dims", where, int)
    if dims <= 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{WHO}: {where}.dims must be even, positive and at most the size it rotates")
    if not _need(rot, "base", where) > 1:
        raise ConfigError(f"{WHO}: {where}.base must be beyond 1")
    sc = rot.get("scaling")
    if sc is None:
        return
    if not scaled:
        raise ConfigError(f"{WHO}: {where}.scaling is not part of this kind of layer")
    for k in ("factor", "low", "high", "original"):
        if not _need(sc, k, where + ".scaling") > 0:
            raise ConfigError(f"{WHO}: {where}.scaling.{k} must be positive")
    if sc["low"] > sc["high"]:
        raise ConfigError(f"{WHO}: {where}.scaling.low exceeds high")


def _check_parallel(m: Any, where: str) -> None:
    left, right = (m or {}).get("left"), (m or {}).get("right")
    _positive(left, ("heads", "kv_heads", "dim", "vdim"), where + ".left")
    if left["heads"] % left["kv_heads"]:
        raise ConfigError(f"{WHO}: {where}.left.heads must be a multiple of kv_heads")
    if not _need(left, "scale", where + ".left") > 0:
        raise ConfigError(f"{WHO}: {where}.left.scale must be positive")
    if left.get("softcap") is not None and _need(left, "softcap", where + ".left") < 0:
        raise ConfigError(f"{WHO}: {where}.left.softcap cannot be negative")
    _check_rot(left.get("rot"), left["dim"], where + ".left.rot", True)
    _positive(right, ("heads", "kv_heads", "dim", "vdim", "conv"), where + ".right")
    if right["heads"] % right["kv_heads"]:
        raise ConfigError(f"{WHO}: {where}.right.heads must be a multiple of kv_heads")
    for k in ("left_scale", "right_scale"):
        _need(m, k, where)


def _check_latent(m: Any, where: str) -> None:
    _positive(m, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), where)
    if not _need(m, "scale", where) > 0:
        raise ConfigError(f"{WHO}: {where}.scale must be positive")
    if m.get("mask") is not None:
        _positive(m["mask"], ("size",), where + ".mask")
    _check_rot(m.get("rot"), m["rot_dim"], where + ".rot", False)


def _check_kv_from(layers, i: int, where: str) -> None:
    m = layers[i]["mixer"]
    j = m.get("kv_from")
    if j is None:
        return
    j = _need(m, "kv_from", where, int)
    if not 0 <= j < i or layers[j]["type"] != "latent_attention" or layers[j]["mixer"].get("kv_from") is not None:
        raise ConfigError(f"{WHO}: {where}.kv_from is {j}; it must name an earlier latent_attention layer that has latents "
                          f"of its own")
    src = layers[j]["mixer"]
    for k in ("kv_rank", "rot_dim", "rot"):
        if src[k] != m[k]:
            raise ConfigError(f"{WHO}: {where}.{k} differs from that of layer {j}, whose latents it reads")


@dataclasses.dataclass
class PapusunConfig(ModelConfig):
    architecture: ClassVar[str] = "Papusun"
    model_types: ClassVar[tuple[str, ...]] = ("papusun",)

    vocab: int = 0
    width: int = 0
    layers: tuple = ()
    norm: Optional[dict] = None
    token_side: Optional[dict] = None
    logit_scale: Optional[float] = None

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
        _positive(self.token_side, ("dim",), "token_side")
        _need({"logit_scale": self.logit_scale}, "logit_scale", "config.json")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, dict) else layer
            if kind not in LAYER_TYPES:
                raise ConfigError(f"{WHO}: {where}.type is {kind!r}; known: {LAYER_TYPES}")
            if kind == "parallel":
                _check_parallel(layer.get("mixer"), where + ".mixer")
            else:
                _check_latent(layer.get("mixer"), where + ".mixer")
                _check_kv_from(self.layers, i, where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"{WHO}: {where}.mlp.kind must be 'dense'")
                _positive(mlp, ("ff",), where + ".mlp")

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def side_dim(self) -> int:
        return int(self.token_side["dim"])
