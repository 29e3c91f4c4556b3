"""Routed feed-forward (mixture of experts) with sigmoid scores and group-limited choice.

Per token, with h its normed input:  s = sigmoid(Wr h) in float32;  choice = s + correction;  the experts come in
``n_groups`` equal groups of neighbours, a group's score is the sum of its two largest choices, and only experts of
the best ``keep_groups`` groups can be chosen (the others count as minus infinity);  the ``top`` largest choices
are taken;  their weights are s (without the correction) times ``scale``, not renormalised.
Expert e is Wdown_e gelu(Wup_e h) with the exact (erf) GELU and no biases;  the output is the weighted sum.

The experts' matrices are stacked at load ([E, ff, d] and [E, d, ff]); a step sorts its (token, choice) rows by
expert on the device and runs one grouped product per projection over them (``ops.moe_experts``)."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops
from ..profiler import bucket
from .base import FEED_FORWARDS, FeedForward, ParamSpec, Runtime, register_part
from .mlp import SwiGLU


@register_part(FEED_FORWARDS, "routed_gelu")
class RoutedGelu(FeedForward):
    graph_safe = True

    def __init__(self, runtime: Runtime, dim: int, intermediate: int, n_experts: int, top: int, scale: float = 1.0,
                 n_groups: int = 1, keep_groups: int = 1, correction: bool = True):
        self.runtime, self.dim, self.intermediate = runtime, int(dim), int(intermediate)
        self.n_experts, self.top, self.scale = int(n_experts), int(top), float(scale)
        self.n_groups, self.keep_groups, self.correction = int(n_groups), int(keep_groups), bool(correction)
        E, G = self.n_experts, self.n_groups
        if not (0 < self.top <= E and G > 0 and E % G == 0 and 0 < self.keep_groups <= G
                and self.keep_groups * (E // G) >= self.top):
            raise ValueError(f"routing of {self.top} of {E} experts in {G} groups keeping {self.keep_groups} is not possible")

    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"router": ParamSpec((self.n_experts, self.dim))}
        if self.correction:
            specs["correction"] = ParamSpec((self.n_experts,), role="vector")
        for e in range(self.n_experts):
            specs[f"up{e}"] = ParamSpec((self.intermediate, self.dim))
            specs[f"down{e}"] = ParamSpec((self.dim, self.intermediate))
        return specs

    def bind(self, params):
        if torch.device(self.runtime.device).type == "cuda":
            ops.require("moe")                    # the kernels of csrc/moe.cu
        self.w_router = params["router"].contiguous()
        self.b_correction = params["correction"].contiguous() if self.correction else None
        self.w_up = torch.stack([params[f"up{e}"] for e in range(self.n_experts)]).contiguous()
        self.w_down = torch.stack([params[f"down{e}"] for e in range(self.n_experts)]).contiguous()

    def forward(self, x, ctx):
        with bucket("mlp.router"):
            ids, wts = ops.moe_route(x, self.w_router, self.b_correction, self.n_groups, self.keep_groups, self.top,
                                     self.scale)
        with bucket("mlp.experts"):
            return ops.moe_experts(x, ids, wts, self.w_up, self.w_down, x.dtype)


@register_part(FEED_FORWARDS, "routed_glu")
class RoutedGLU(FeedForward):
    """Routed gated experts.  z = Wr h + b in float32, and by ``scores``

    * "softmax_top": the ``top`` experts of largest z are taken and weighted by the softmax over those logits alone;
    * "softmax": s = softmax(z) over all experts; the experts come in ``n_groups`` equal groups of neighbours whose score
      is their largest s, only experts of the best ``keep_groups`` groups can be chosen, the ``top`` largest s are taken
      and weighted by s divided by the sum over the chosen.  ``correction``: a learned number per expert is added to s for
      the choice (and for the groups), not for the weights.

    Expert e is Wdown_e (silu(Wgate_e h) * (Wup_e h)), no biases; the output is the weighted sum.  ``shared`` > 0: one
    more expert of that inner size runs for every token and is added; ``shared_gate``: times sigmoid(w h), one number per
    token, whose row w rides in the router's product.  ``identity`` more experts have no tensors: such an expert's result is
    h itself.  [gate; up] of every expert is one stacked matrix, so the first grouped product gives both halves."""
    graph_safe = True

    def __init__(self, runtime: Runtime, dim: int, intermediate: int, n_experts: int, top: int, bias: bool = True,
                 scores: str = "softmax_top", n_groups: int = 1, keep_groups: int = 1, shared: int = 0,
                 correction: bool = False, identity: int = 0, shared_gate: bool = False):
        self.runtime, self.dim, self.intermediate = runtime, int(dim), int(intermediate)
        self.n_experts, self.top, self.bias = int(n_experts), int(top), bool(bias)
        self.scores, self.n_groups, self.keep_groups = scores, int(n_groups), int(keep_groups)
        if scores not in ("softmax_top", "softmax"):
            raise ValueError(f"router scores {scores!r} are not known ('softmax_top', 'softmax')")
        self.correction, self.identity, self.shared_gate = bool(correction), int(identity), bool(shared_gate)
        E = self.n_choices = self.n_experts + self.identity
        if not (0 < self.top <= E and self.n_experts > 0 and self.identity >= 0):
            raise ValueError(f"cannot choose {top} of {n_experts} experts and {identity} identity experts")
        if (self.correction and scores != "softmax") or (self.shared_gate and not shared):
            raise ValueError("a correction needs softmax scores, a gate of the shared expert a shared expert")
        G = self.n_groups
        if not (G > 0 and E % G == 0 and 0 < self.keep_groups <= G
                and self.keep_groups * (E // G) >= self.top) or (G > 1 and scores != "softmax"):
            raise ValueError(f"routing of {top} of {n_experts} experts in {G} groups keeping {keep_groups} is not possible")
        if scores == "softmax" and self.bias:
            raise ValueError("softmax scores take no bias")
        self.shared = SwiGLU(runtime, dim, shared) if shared else None

    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"router": ParamSpec((self.n_choices, self.dim))}
        if self.bias:
            specs["router_bias"] = ParamSpec((self.n_choices,), role="vector")
        if self.correction:
            specs["correction"] = ParamSpec((self.n_choices,), role="vector")
        if self.shared_gate:
            specs["shared_gate"] = ParamSpec((1, self.dim))
        for e in range(self.n_experts):
            specs[f"gate{e}"] = ParamSpec((self.intermediate, self.dim))
            specs[f"up{e}"] = ParamSpec((self.intermediate, self.dim))
            specs[f"down{e}"] = ParamSpec((self.dim, self.intermediate))
        if self.shared is not None:
            specs.update({"shared." + k: v for k, v in self.shared.param_specs().items()})
        return specs

    def bind(self, params):
        if torch.device(self.runtime.device).type == "cuda":
            ops.require("moe")                    # the kernels of csrc/moe.cu
        rows = [params["router"]] + ([params["shared_gate"]] if self.shared_gate else [])
        self.w_router = torch.cat(rows, dim=0).contiguous()
        self.b_router = params["router_bias"].contiguous() if self.bias else None
        self.b_correction = params["correction"].contiguous() if self.correction else None
        self.w_up = torch.stack([torch.cat([params[f"gate{e}"], params[f"up{e}"]], dim=0)
                                 for e in range(self.n_experts)]).contiguous()               # [E, 2 ff, d]
        self.w_down = torch.stack([params[f"down{e}"] for e in range(self.n_experts)]).contiguous()
        if self.shared is not None:
            self.shared.bind({k[7:]: v for k, v in params.items() if k.startswith("shared.")})

    def forward(self, x, ctx):
        with bucket("mlp.router"):
            extra = int(self.shared_gate)
            if self.scores == "softmax":
                ids, wts, *gate = ops.moe_route(x, self.w_router, self.b_correction, self.n_groups, self.keep_groups, self.top,
                                                1.0, softmax=True, group_max=True, renormalise=True, extra_rows=extra)
            else:
                ids, wts, *gate = ops.moe_route(x, self.w_router, self.b_router, 1, 1, self.top, 1.0, softmax_top=True,
                                                extra_rows=extra)
        shared = self.shared.forward(x, ctx) if self.shared is not None else None
        with bucket("mlp.experts"):
            return ops.moe_experts(x, ids, wts, self.w_up, self.w_down, x.dtype, glu=True, add=shared,
                                   add_gate=gate[0] if gate else None, identity=self.identity > 0)
