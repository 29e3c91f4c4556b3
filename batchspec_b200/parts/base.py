"""Interfaces of the parts a decoder is assembled from, and their registries.

A *part* is a parametrised object that knows its own sizes and constants and
nothing about the model it sits in: it names its tensors by short local names
(``q``, ``gate`` ...), the architecture supplies the map from local names to
checkpoint names.  The reference fixes the parts by subclass hooks
(batchspec/models/base_model.py:138-173, ``_get_attention_class`` /
``_get_block_class``); here they are chosen per layer by the model description, so
one model may mix different mixers and feed-forwards.

Registries: ``MIXERS``, ``FEED_FORWARDS``, ``NORMS``, ``POSITION_ENCODINGS``,
``BLOCKS``, ``BRANCH_SCALES``, ``STREAM_MIXES``, ``DEPTH_AVERAGES``, ``INPUT_PARTS``, ``LOGITS_PARTS``.  ``register_part(registry, kind)``
is a class decorator; ``build_part(registry, spec, runtime)`` instantiates
``spec.kind`` with ``spec.params``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

import torch


@dataclass(frozen=True)
class PartSpec:
    """Which part (``kind``) and with which sizes/constants (``params``)."""
    kind: str
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class ParamSpec:
    """One tensor a part needs.

    role: ``matrix`` (a GEMM operand or lookup table: held in the run dtype),
          ``vector`` (a per-channel scale: held in the run dtype unless the file
          stores it in 32-bit, which is kept), ``int`` (an integer table: int32).
    init: ``normal`` -> N(0, std);  ``ones_normal`` -> 1 + N(0, std).
    """
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"


@dataclass(frozen=True)
class CacheSpec:
    """What a mixer asks of the paged cache, per token and per layer.

    policy ``full``: every token's entry is kept while the request lives.
    policy ``window``: only the last ``window`` tokens are ever read; pages that
    lie wholly before the window are given back.
    policy ``chunk``: a token reads only the tokens of its own chunk of ``window``
    positions (counted from position 0); pages that lie wholly before the chunk of
    the next position are given back.
    ``entry_shape`` is the per-token shape of ONE stored tensor, e.g.
    (n_kv_heads, head_dim); ``tensors`` says how many of them a token has: 2 for
    keys and values, 1 for a mixer that stores a single (compressed) entry.
    ``page_size``: tokens per page of this mixer's group, or None for the
    engine's default; groups with different page sizes have block tables of
    different lengths for the same request.
    ``pool`` P > 0: besides, every whole block of P tokens has one more entry of the
    same shape, which is kept while the request lives.  These entries have a group of
    their own (pages of as many entries, a block table: entry b is block b), and a
    windowed group keeps the tokens of the block that is not yet whole.
    ``keep``: with policy ``window``, the request's first ``keep`` tokens are read however far the window has moved;
    their pages are not given back."""
    policy: str
    entry_shape: Tuple[int, ...]
    window: Optional[int] = None
    tensors: int = 2
    page_size: Optional[int] = None
    pool: int = 0
    keep: int = 0


@dataclass(frozen=True)
class StateSpec:
    """Fixed-size per-request state of a mixer (a recurrent state, a conv tail):
    one tensor of ``shape``/``dtype`` per live request, zeroed when a request is
    admitted, addressed by the request's state slot."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class Runtime:
    """What every part gets at construction: run dtype and device."""
    dtype: torch.dtype
    device: torch.device


class Part:
    """Common protocol.  ``param_specs`` -> local name -> ParamSpec;
    ``bind`` receives the loaded tensors (on the device) under those names.
    ``graph_safe``: True if ``forward`` only enqueues device work whose launch
    sizes depend on the number of tokens and entries alone and reads everything
    else from the step context's device tensors; such parts may be captured in a
    CUDA graph.  A part that reads host fields of the context must leave it False."""
    graph_safe = False

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {}

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        pass


class Norm(Part):
    """``forward(resid, delta, delta_scale=1.0, delta_vec=None)``: ``resid`` is the float32 residual
    stream [n, d]; if ``delta`` is given, ``delta_scale * delta`` (times ``delta_vec``, a float32 factor per
    column, when a block scales its branches that way) is first added into
    ``resid`` in place (the residual sum, in 32-bit); returns the normalised rows in
    the run dtype."""

    def forward(self, resid: torch.Tensor, delta: Optional[torch.Tensor], delta_scale: float = 1.0,
                delta_vec: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class PositionEncoding(Part):
    """``apply(q, k, ctx)`` rotates/offsets q [n, Hq, hd] and k [n, Hkv, hd] (views,
    in place) for the tokens' absolute positions ``ctx.positions``.  A part that
    can be folded into the attention mixer's fused rotate-and-append kernel also
    offers ``rope_table()`` -> (``ops.rope_frequency_table`` of rotary_dim/2 frequencies, rotary_dim,
    interleaved)."""

    def apply(self, q: torch.Tensor, k: torch.Tensor, ctx) -> None:
        raise NotImplementedError

    def rope_table(self):
        return None


class Mixer(Part):
    """Token mixer.  ``forward(x, ctx, cache)``: x [n, d] run dtype -> [n, d].
    ``cache`` is the LayerCache the model description assigned to this run of the
    layer (None if the mixer declared no needs): ``cache.kv`` the layer's page
    tensor and ``cache.group`` the index of its block tables in ``ctx``,
    ``cache.state`` its per-request state tensor [max_requests, *shape],
    ``cache.owner`` False when the layer only reads another layer's cache;
    ``cache.pooled`` and ``cache.pooled_group`` the pages and the group of the blocks'
    entries (a spec with ``pool``)."""

    def cache_spec(self) -> Optional[CacheSpec]:
        return None

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    """``forward(x, ctx)``: x [n, d] run dtype -> [n, d]."""

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        raise NotImplementedError


class InputPart(Part):
    """Runs once per step right after the embedding: ``forward(resid, ctx)`` changes
    the float32 residual rows [n, d] in place (a learned absolute position row
    added to each token, a multiplier ...).  A part that keeps something per request from step to step (the
    request's last token, say) declares it with ``state_spec()`` and receives the tensor [slots, *shape] as
    ``state``; it is zeroed when a request is admitted and indexed by ``ctx.state_slots``."""

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def forward(self, resid: torch.Tensor, ctx, state: Optional[torch.Tensor] = None) -> None:
        raise NotImplementedError


class LogitsPart(Part):
    """Runs once per step on the head's output: ``forward(logits, ctx)`` changes the
    float32 logits [wanted rows, vocab] in place (a scale, a soft cap ...)."""

    def forward(self, logits: torch.Tensor, ctx) -> None:
        raise NotImplementedError


MIXERS: Dict[str, type] = {}
FEED_FORWARDS: Dict[str, type] = {}
NORMS: Dict[str, type] = {}
POSITION_ENCODINGS: Dict[str, type] = {}
BLOCKS: Dict[str, type] = {}
BRANCH_SCALES: Dict[str, type] = {}
STREAM_MIXES: Dict[str, type] = {}
DEPTH_AVERAGES: Dict[str, type] = {}
INPUT_PARTS: Dict[str, type] = {}
LOGITS_PARTS: Dict[str, type] = {}


@dataclass
class BranchJoin:
    """How a branch y joins the residual x when it is normed on its way: x + y / rms(y) * ``post`` (float32 [d]; rms
    with ``eps``), and then, with ``coef`` (float32 [j + 1]), the average sum_{i < j} coef[i] X_i + coef[j] x over the
    residuals X_i that went into the layers so far, which the executor keeps (``ModelSpec.depth_average``)."""
    post: Optional[torch.Tensor] = None
    eps: float = 0.0
    coef: Optional[torch.Tensor] = None


class Block:
    """Arrangement of a layer's parts around the residual stream.  A block kind
    declares its slots as data: ``SLOTS`` maps slot name -> the registry its part
    comes from, in the order the parts' tensors are listed; the model description
    gives one ``PartSpec`` per slot.  ``MIXER_SLOT`` names the slot whose part
    (a ``Mixer``) owns the layer's cache and per-request state.  The built parts
    arrive as keyword arguments and are kept as attributes of the same names and in
    ``self.parts``.

    ``forward(resid, pending, ctx, cache, pending_scale=1.0)`` takes the float32 residual and a
    not-yet-added branch output (or None) with the factor it is to be added with, and returns the
    residual and its own last branch output, so the add can be fused into the next norm.  ``residual_mult``
    is the factor of the branch a block returns; a block that also multiplies that branch by a learned factor per
    column has it (float32 [d]) in ``residual_vec``, and whoever adds the branch applies both (the next block gets
    the vector as ``pending_vec``).  A block of a model that keeps several residual streams per token gets them as
    ``resid`` [n, S, d]; the coefficients with which its last branch joins the streams are its ``residual_mix``
    (float32 [S * S + S]: the mix matrix indexed (from, to), then the factor of the branch per stream), handed on as
    ``pending_mix``.  A block whose branches are normed before they join says so in ``residual_join`` (a ``BranchJoin``),
    handed on as ``pending_join``; in a model that averages over depth its forward also takes ``history`` (float32
    [layer runs + 1, n, d]) and ``slot``: the residual that enters the run is stored as history[slot]."""
    SLOTS: Dict[str, Dict[str, type]] = {}
    MIXER_SLOT = "mixer"
    residual_mult = 1.0
    residual_vec = None
    residual_mix = None
    residual_join = None

    def __init__(self, **parts):
        missing, extra = set(self.SLOTS) - set(parts), set(parts) - set(self.SLOTS)
        if missing or extra:
            raise ValueError(f"block {type(self).__name__} has slots {list(self.SLOTS)}; missing {sorted(missing)}, "
                             f"unexpected {sorted(extra)}")
        self.parts = {slot: parts[slot] for slot in self.SLOTS}
        for slot, part in self.parts.items():
            setattr(self, slot, part)

    def forward(self, resid, pending, ctx, cache, pending_scale: float = 1.0):
        raise NotImplementedError


def register_part(registry: Dict[str, type], kind: str):
    def deco(cls):
        registry[kind] = cls
        cls.kind = kind
        return cls
    return deco


def build_part(registry: Dict[str, type], spec: PartSpec, runtime: Runtime):
    if spec.kind not in registry:
        raise KeyError(f"part kind {spec.kind!r} is not registered (known: {sorted(registry)})")
    return registry[spec.kind](runtime=runtime, **spec.params)
