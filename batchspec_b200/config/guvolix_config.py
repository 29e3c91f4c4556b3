"""Configuration of the Guvolix design: a decoder whose ``config.json`` lists its layers one by one.

    {"architecture": "Guvolix", "vocab": V, "width": d, "norm": {"eps": e}, "embedding": {"scale": m},
     "layers": [{"type": "parallel" | "parallel_2", "mixer": {"left": {...}, "right": {...}, ...},
                 "mlp": {"kind": "dense", "ff": F} | {"kind": "moe", ...} | null}, ...]}

``left`` is the same in both types: heads, kv_heads, dim, vdim, scale, ``rot`` {base, dims, scaling} and ``mask`` {size,
keep_first}: a sliding window and how many first tokens stay visible behind it.  ``rot.scaling`` is {factor}, or {factor,
low, high, original} for frequencies scaled by their wavelength.  The ``right`` of a ``parallel`` mixer gives heads, vdim,
state, groups, conv and norm_groups (a state space recurrence), that of a ``parallel_2`` mixer heads, dim, vdim and
gate_cap (a matrix memory), beside left_scale and right_scale.  A routed feed-forward gives ``expert`` {ff}, ``router``
{experts, identity, top} and ``shared`` {ff}.  Absent rot, scaling, mask, keep_first, identity, shared and mlp mean none.
Every size and constant is read from here; keys this reader does not know are listed in ``unread_keys``."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .model_config import ConfigError, _take, register_config_class

_TOP = {"architecture", "architectures", "vocab", "width", "norm", "embedding", "layers"}
_LEFT = {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"}
_STATE_SPACE = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
_MATRIX_MEMORY = ("heads", "dim", "vdim")


def _unknown(d: Dict[str, Any], known, where: str, out: List[str]) -> None:
    out.extend(f"{where}{k}" for k in sorted(set(d) - set(known)))


def _positive(d: Dict[str, Any], keys, where: str) -> None:
    for key in keys:
        if _take(d, key, int) <= 0:
            raise ConfigError(f"config.json: {where}.{key} must be positive")


def _attention(m: Dict[str, Any], where: str, unread: List[str]) -> None:
    _unknown(m, _LEFT, where + ".", unread)
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _take(m, "scale", float)
    mask = m.get("mask")
    if mask is not None:
        _unknown(mask, {"size", "keep_first"}, where + ".mask.", unread)
        _positive(mask, ("size",), where + ".mask")
        if _take(mask, "keep_first", int, 0) < 0:
            raise ConfigError(f"config.json: {where}.mask.keep_first must not be negative")
    rot = m.get("rot")
    if rot is None:
        return
    _unknown(rot, {"base", "dims", "scaling"}, where + ".rot.", unread)
    dims = _take(rot, "dims", int)
    if not _take(rot, "base", float) > 0 or dims < 0 or dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}.rot needs a positive base and an even number of dims, at most dim")
    scaling = rot.get("scaling")
    if scaling:
        ramp = {"low", "high", "original"} if "original" in scaling else set()
        _unknown(scaling, {"factor"} | ramp, where + ".rot.scaling.", unread)
        if not all(_take(scaling, key, float) > 0 for key in {"factor"} | ramp) or (ramp and scaling["low"] == scaling["high"]):
            raise ConfigError(f"config.json: {where}.rot.scaling needs positive numbers, low and high different")


def _feed_forward(f: Optional[Dict[str, Any]], where: str, unread: List[str]) -> None:
    if f is None:
        return
    kind = f.get("kind")
    if kind == "dense":
        _unknown(f, {"kind", "ff"}, where + ".", unread)
        _positive(f, ("ff",), where)
        return
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not known ('dense', 'moe', or null for no feed-forward)")
    _unknown(f, {"kind", "expert", "router", "shared"}, where + ".", unread)
    expert, router, shared = f.get("expert") or {}, f.get("router") or {}, f.get("shared")
    _unknown(expert, {"ff"}, where + ".expert.", unread)
    _positive(expert, ("ff",), where + ".expert")
    _unknown(router, {"experts", "identity", "top"}, where + ".router.", unread)
    _positive(router, ("experts", "top"), where + ".router")
    identity = _take(router, "identity", int, 0)
    if identity < 0 or router["top"] > router["experts"] + identity:
        raise ConfigError(f"config.json: {where}.router: {router['top']} of {router['experts']} experts and {identity} "
                          f"identity experts is not possible")
    if shared is not None:
        _unknown(shared, {"ff"}, where + ".shared.", unread)
        _positive(shared, ("ff",), where + ".shared")


@dataclass(frozen=True)
class GuvolixConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    embed_scale: float
    layers: Tuple[Dict[str, Any], ...]
    unread_keys: Tuple[str, ...] = ()

    @classmethod
    def from_json_dict(cls, d: Dict[str, Any]) -> "GuvolixConfig":
        unread: List[str] = []
        _unknown(d, _TOP, "", unread)
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        norm, emb = d.get("norm") or {}, d.get("embedding") or {}
        _unknown(norm, {"eps"}, "norm.", unread)
        _unknown(emb, {"scale"}, "embedding.", unread)
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            _unknown(layer, {"type", "mixer", "mlp"}, where + ".", unread)
            kind, m, at = layer.get("type"), layer.get("mixer") or {}, where + ".mixer"
            left, right = m.get("left") or {}, m.get("right") or {}
            if kind == "parallel":
                _unknown(m, {"left", "right"}, at + ".", unread)
                _unknown(right, _STATE_SPACE, at + ".right.", unread)
                _positive(right, _STATE_SPACE, at + ".right")
                if right["heads"] % right["groups"] or (right["heads"] * right["vdim"]) % right["norm_groups"]:
                    raise ConfigError(f"config.json: {at}.right: groups must divide heads, and norm_groups heads * vdim")
            elif kind == "parallel_2":
                _unknown(m, {"left", "right", "left_scale", "right_scale"}, at + ".", unread)
                _unknown(right, _MATRIX_MEMORY + ("gate_cap",), at + ".right.", unread)
                _positive(right, _MATRIX_MEMORY, at + ".right")
                if not _take(right, "gate_cap", float) > 0:
                    raise ConfigError(f"config.json: {at}.right.gate_cap must be positive")
                _take(m, "left_scale", float)
                _take(m, "right_scale", float)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design "
                                  f"(known: 'parallel', 'parallel_2')")
            _attention(left, at + ".left", unread)
            _feed_forward(layer.get("mlp"), where + ".mlp", unread)
        cfg = cls(architecture=d.get("architecture") or (d.get("architectures") or [None])[0],
                  vocab_size=_take(d, "vocab", int), width=_take(d, "width", int), norm_eps=_take(norm, "eps", float),
                  embed_scale=_take(emb, "scale", float, 1.0), layers=tuple(copy.deepcopy(layers)),
                  unread_keys=tuple(unread))
        if cfg.vocab_size <= 0 or cfg.width <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: vocab and width must be positive and norm.eps > 0")
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale},
                "layers": copy.deepcopy(list(self.layers))}


register_config_class("Guvolix", GuvolixConfig)
