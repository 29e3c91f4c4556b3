"""Configuration of the Podizen design: a decoder whose ``config.json`` lists its layers one by one.

    {"architecture": "Podizen", "vocab": V, "width": d, "norm": {"eps": e},
     "layers": [{"type": "attention" | "parallel", "mixer": {...}, "mlp": {"kind": "moe", ...} | null}, ...]}

An ``attention`` mixer gives heads, kv_heads, dim, vdim, scale and ``mask`` {size}: a sliding window.  A ``parallel``
mixer gives ``left`` (the same, with ``mask`` {size, pool}: a window and blocks of ``pool`` tokens before it, and ``rot``
{base, dims}) and ``right`` (heads, dim, vdim, decay: a factor per head, ``rot``).  A feed-forward gives ``expert`` {ff},
``router`` {experts, top, groups {count, keep}} and ``shared`` {ff}.  Absent mask, pool, rot, groups and shared mean
none.  Every size and constant is read from here; keys this reader does not know are listed in ``unread_keys``."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .model_config import ConfigError, _take, register_config_class

_TOP = {"architecture", "architectures", "vocab", "width", "norm", "layers"}
_ATTENTION = {"heads", "kv_heads", "dim", "vdim", "scale", "mask"}
_RIGHT = {"heads", "dim", "vdim", "decay", "rot"}


def _unknown(d: Dict[str, Any], known, where: str, out: List[str]) -> None:
    out.extend(f"{where}{k}" for k in sorted(set(d) - set(known)))


def _positive(d: Dict[str, Any], keys, where: str) -> None:
    for key in keys:
        if _take(d, key, int) <= 0:
            raise ConfigError(f"config.json: {where}.{key} must be positive")


def _rotation(m: Dict[str, Any], where: str, unread: List[str]) -> None:
    rot = m.get("rot")
    if rot is not None:
        _unknown(rot, {"base", "dims"}, where + ".rot.", unread)
        dims = _take(rot, "dims", int)
        if not _take(rot, "base", float) > 0 or dims < 0 or dims % 2 or dims > m["dim"]:
            raise ConfigError(f"config.json: {where}.rot needs a positive base and an even number of dims, at most dim")


def _softmax_mixer(m: Dict[str, Any], where: str, pool: bool, unread: List[str]) -> None:
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _take(m, "scale", float)
    mask = m.get("mask")
    if mask is not None:
        _unknown(mask, {"size", "pool"} if pool else {"size"}, where + ".mask.", unread)
        _positive(mask, ("size", "pool") if mask.get("pool") is not None and pool else ("size",), where + ".mask")


def _feed_forward(f: Optional[Dict[str, Any]], where: str, unread: List[str]) -> None:
    if f is None:
        return
    if f.get("kind", "moe") != "moe":
        raise ConfigError(f"config.json: {where}.kind {f.get('kind')!r} is not known ('moe', or null for no feed-forward)")
    _unknown(f, {"kind", "expert", "router", "shared"}, where + ".", unread)
    expert, router, shared = f.get("expert") or {}, f.get("router") or {}, f.get("shared")
    _unknown(expert, {"ff"}, where + ".expert.", unread)
    _positive(expert, ("ff",), where + ".expert")
    _unknown(router, {"experts", "top", "groups"}, where + ".router.", unread)
    _positive(router, ("experts", "top"), where + ".router")
    groups = router.get("groups") or {"count": 1, "keep": 1}
    _unknown(groups, {"count", "keep"}, where + ".router.groups.", unread)
    _positive(groups, ("count", "keep"), where + ".router.groups")
    E, count, keep = router["experts"], groups["count"], groups["keep"]
    if E % count or keep > count or keep * (E // count) < router["top"]:
        raise ConfigError(f"config.json: {where}.router: {router['top']} of {E} experts in {count} groups of which {keep} "
                          f"are kept is not possible")
    if shared is not None:
        _unknown(shared, {"ff"}, where + ".shared.", unread)
        _positive(shared, ("ff",), where + ".shared")


@dataclass(frozen=True)
class PodizenConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    unread_keys: Tuple[str, ...] = ()

    @classmethod
    def from_json_dict(cls, d: Dict[str, Any]) -> "PodizenConfig":
        unread: List[str] = []
        _unknown(d, _TOP, "", unread)
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        norm = d.get("norm") or {}
        _unknown(norm, {"eps"}, "norm.", unread)
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            _unknown(layer, {"type", "mixer", "mlp"}, where + ".", unread)
            kind, m, at = layer.get("type"), layer.get("mixer") or {}, where + ".mixer"
            if kind == "attention":
                _unknown(m, _ATTENTION, at + ".", unread)
                _softmax_mixer(m, at, False, unread)
            elif kind == "parallel":
                _unknown(m, {"left", "right"}, at + ".", unread)
                left, right = m.get("left") or {}, m.get("right") or {}
                _unknown(left, _ATTENTION | {"rot"}, at + ".left.", unread)
                _softmax_mixer(left, at + ".left", True, unread)
                _rotation(left, at + ".left", unread)
                _unknown(right, _RIGHT, at + ".right.", unread)
                _positive(right, ("heads", "dim", "vdim"), at + ".right")
                _rotation(right, at + ".right", unread)
                decay = right.get("decay")
                if not isinstance(decay, list) or len(decay) != right["heads"] or \
                        not all(isinstance(x, (int, float)) and not isinstance(x, bool) for x in decay):
                    raise ConfigError(f"config.json: {at}.right.decay must list one number per head")
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design "
                                  f"(known: 'attention', 'parallel')")
            _feed_forward(layer.get("mlp"), where + ".mlp", unread)
        cfg = cls(architecture=d.get("architecture") or (d.get("architectures") or [None])[0],
                  vocab_size=_take(d, "vocab", int), width=_take(d, "width", int), norm_eps=_take(norm, "eps", float),
                  layers=tuple(copy.deepcopy(layers)), unread_keys=tuple(unread))
        if cfg.vocab_size <= 0 or cfg.width <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: vocab and width must be positive and norm.eps > 0")
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}


register_config_class("Podizen", PodizenConfig)
