"""Generic executor of a ``ModelSpec``: embedding (then the optional input part),
the listed runs of layers, final norm, head over the wanted rows only (then the
optional logits part).

The reference computes logits for every token of the step and then selects the
last row of each request (batchspec/models/standard_model.py:90-102,
backends/standard_engine.py:127); here only the rows asked for reach the head."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..kernels import ops
from ..profiler import bucket
from ..parts.base import (BLOCKS, INPUT_PARTS, LOGITS_PARTS, NORMS, CacheSpec, ParamSpec, Runtime, StateSpec,
                          build_part)
from .spec import ModelSpec


@dataclass
class LayerCache:
    """What one run of a layer sees of the cache.  ``kv``: [pages, tensors per token,
    page_size * entry elements] of its group's pool (None if the mixer asked for no pages);
    ``group``: index of the block tables in the step context; ``state``:
    [max_requests, *state_shape] or None; ``owner``: False for a run that reads
    another run's cache.  ``pooled`` / ``pooled_group``: the same two for the entries of
    pooled blocks, if the mixer asked for them."""
    kv: Optional[torch.Tensor]
    group: int
    state: Optional[torch.Tensor]
    owner: bool
    pooled: Optional[torch.Tensor] = None
    pooled_group: int = -1


@dataclass
class CacheNeed:
    """Per run of the order: what its mixer asks for and whose cache it uses."""
    cache: Optional[CacheSpec]
    state: Optional[StateSpec]
    cache_from: Optional[int]


class DecoderModel:
    def __init__(self, spec: ModelSpec, runtime: Runtime):
        self.spec, self.runtime = spec, runtime
        self.blocks = []
        for i, layer in enumerate(spec.layers):
            if layer.block not in BLOCKS:
                raise KeyError(f"block kind {layer.block!r} is not registered (known: {sorted(BLOCKS)})")
            kind = BLOCKS[layer.block]
            if set(layer.parts) != set(kind.SLOTS):
                raise ValueError(f"layer {i}: block {layer.block!r} has slots {list(kind.SLOTS)}, "
                                 f"the description gives {list(layer.parts)}")
            self.blocks.append(kind(**{slot: build_part(registry, layer.parts[slot], runtime)
                                       for slot, registry in kind.SLOTS.items()}, **layer.block_params))
        self.final_norm = build_part(NORMS, spec.final_norm, runtime)
        self.input_part = build_part(INPUT_PARTS, spec.input_part, runtime) if spec.input_part else None
        self.logits_part = build_part(LOGITS_PARTS, spec.logits_part, runtime) if spec.logits_part else None
        for e, run in enumerate(spec.order):
            if not 0 <= run.layer < len(spec.layers):
                raise ValueError(f"order[{e}] names layer {run.layer}, the model has {len(spec.layers)}")
            if run.cache_from is not None:
                if not 0 <= run.cache_from < e or spec.order[run.cache_from].cache_from is not None:
                    raise ValueError(f"order[{e}].cache_from must name an earlier run that owns its cache")
        self.embed: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.caches: List[Optional[LayerCache]] = [None] * len(spec.order)
        self.input_state: Optional[torch.Tensor] = None      # the input part's per-request state, if it declared one
        # debugging aid: called as probe(run index, residual after the run, float32 [n, d]) when set
        self.layer_probe = None

    @property
    def graph_safe(self) -> bool:
        parts = [self.final_norm, self.input_part, self.logits_part]
        for b in self.blocks:
            for part in b.parts.values():
                parts += [part, getattr(part, "position", None)]
        return all(getattr(p, "graph_safe", False) for p in parts if p is not None)

    # -- tensors ---------------------------------------------------------------
    def _named_parts(self):
        """(what it is, part, local name -> checkpoint name) of every part that holds tensors, in a fixed order."""
        s = self.spec
        if self.input_part is not None:
            yield "input part", self.input_part, s.input_names
        for i, layer in enumerate(s.layers):
            for slot, part in self.blocks[i].parts.items():
                yield f"layer {i}", part, {local: layer.names.get(f"{slot}.{local}") for local in part.param_specs()}, f"{slot}."
        yield "final norm", self.final_norm, s.final_norm_names
        if self.logits_part is not None:
            yield "logits part", self.logits_part, s.logits_names

    def param_specs(self) -> Dict[str, ParamSpec]:
        """checkpoint name -> ParamSpec, in a fixed order."""
        s = self.spec
        out = {s.embed_name: ParamSpec((s.vocab_size, s.hidden_size))}
        for where, part, names, *prefix in self._named_parts():
            for local, ps in part.param_specs().items():
                if names.get(local) is None:
                    raise KeyError(f"{where}: no checkpoint name given for '{(prefix[0] if prefix else '') + local}'")
                out[names[local]] = ps
        if s.lm_head_name is not None:
            out[s.lm_head_name] = ParamSpec((s.vocab_size, s.hidden_size))
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        self.embed = tensors[s.embed_name]
        for where, part, names, *prefix in self._named_parts():
            part.bind({local: tensors[names[local]] for local in part.param_specs()})
        self.head = self.embed if s.lm_head_name is None else tensors[s.lm_head_name]

    # -- cache -----------------------------------------------------------------
    def cache_needs(self) -> List[CacheNeed]:
        """One need per run of the order; after them one more (state only) if the input part keeps something per
        request."""
        out = []
        for run in self.spec.order:
            block = self.blocks[run.layer]
            mixer = getattr(block, block.MIXER_SLOT)
            out.append(CacheNeed(mixer.cache_spec(), mixer.state_spec(), run.cache_from))
        input_state = self.input_part.state_spec() if self.input_part is not None else None
        if input_state is not None:
            out.append(CacheNeed(None, input_state, None))
        return out

    def attach_caches(self, caches: List[Optional[LayerCache]]) -> None:
        n = len(self.spec.order)
        assert len(caches) in (n, n + 1)
        self.caches = list(caches[:n])
        extra = caches[n] if len(caches) > n else None
        self.input_state = extra.state if extra is not None else None

    # -- one step --------------------------------------------------------------
    def forward(self, ctx) -> torch.Tensor:
        """ctx: the step context (token ids, positions, tables, wanted rows).
        Returns float32 logits [len(ctx.logit_rows), vocab]."""
        s = self.spec
        n = ctx.n_tokens
        resid = torch.empty((n, s.hidden_size), dtype=torch.float32, device=self.runtime.device)
        with bucket("embed"):
            ops.embed(ctx.token_ids, self.embed, resid, s.embed_scale)
        if self.input_part is not None:
            if self.input_state is not None:
                self.input_part.forward(resid, ctx, self.input_state)
            else:
                self.input_part.forward(resid, ctx)
        first = resid.clone() if any(run.add_input for run in s.order) else None
        if s.streams:
            if first is not None:
                raise ValueError("a model of several residual streams cannot add its input again before a run")
            # [n, S, d]; the first run's norm fills it from the embedding rows (``expand_from``)
            expand = resid
            resid = torch.empty((n, s.streams, s.hidden_size), dtype=torch.float32, device=self.runtime.device)
        pending, scale, vec, mix, join = None, 1.0, None, None, None
        history = None
        if s.depth_average:
            if first is not None or s.streams:
                raise ValueError("a model that averages over depth has one residual stream and adds no input again")
            history = torch.empty((len(s.order) + 1, n, s.hidden_size), dtype=torch.float32, device=self.runtime.device)
        for e, run in enumerate(s.order):
            if run.add_input:
                if join is not None:
                    raise ValueError("a branch that is normed before it joins cannot be followed by the input again")
                ops.residual_update(resid, pending, scale, first, vec)
                pending, scale, vec = None, 1.0, None
            block = self.blocks[run.layer]
            # a block whose forward knows no branch factors (one registered from outside) can follow any block that
            # leaves its branch unscaled
            extra = {} if scale == 1.0 else {"pending_scale": scale}
            if vec is not None:
                extra["pending_vec"] = vec
            if mix is not None:
                extra["pending_mix"] = mix
            if s.streams and e == 0:
                extra["expand_from"] = expand
            if join is not None:
                extra["pending_join"] = join
            if history is not None:
                extra["history"], extra["slot"] = history, e
            resid, pending = block.forward(resid, pending, ctx, self.caches[e], **extra)
            scale, vec = getattr(block, "residual_mult", 1.0), getattr(block, "residual_vec", None)
            mix, join = getattr(block, "residual_mix", None), getattr(block, "residual_join", None)
            if s.streams and (mix is None or scale != 1.0):
                raise ValueError(f"block kind {block.kind!r} does not keep several residual streams")
            if self.layer_probe is not None:
                if s.streams:
                    after = torch.empty((n, s.hidden_size), dtype=torch.float32, device=self.runtime.device)
                    every = torch.arange(n, dtype=torch.int32, device=self.runtime.device)
                    ops.stream_gather(resid, pending, vec, mix, every, after)
                elif join is not None:
                    after = torch.empty_like(resid)
                    ops.branch_join(resid, pending, dst=after, post=join.post, branch_eps=join.eps, hist=history,
                                    slot=e + 1 if history is not None else 0, coef=join.coef)
                else:
                    after = resid.clone()
                    ops.residual_update(after, pending, scale, vec=vec)
                self.layer_probe(e, after)
        n_out = ctx.n_logit_rows
        if n_out == 0:
            return torch.empty((0, s.vocab_size), dtype=torch.float32, device=self.runtime.device)
        if join is not None:          # the last branch's join, on the wanted rows only, and the final norm in one kernel
            z = self.final_norm.forward_join(resid, pending, join, history, len(s.order) if history is not None else 0,
                                             rows=ctx.logit_rows)
        else:
            picked = torch.empty((n_out, s.hidden_size), dtype=torch.float32, device=self.runtime.device)
            if s.streams:
                ops.stream_gather(resid, pending, vec, mix, ctx.logit_rows, picked)
            else:
                ops.gather_rows_add(resid, pending, ctx.logit_rows, picked, scale, vec)
            z = self.final_norm.forward(picked, None)
        with bucket("lm_head"):
            logits = ops.linear(z, self.head, out_dtype=torch.float32)
        if self.logits_part is not None:
            self.logits_part.forward(logits, ctx)
        return logits
