"""Retention: a decaying [key x value] state per head, read by rotated queries and written by rotated keys.

With h the token's normed input and H heads:

    q, k = Wq h, Wk h   (H x dim, both rotated by position),   v = Wv h   (H x v_dim),   k <- k / sqrt(dim)
    per head:  S <- decay S + k v^T,   o = S^T q         S from zero, a token reads its own write
    out = Wo (concat_heads(o / rms(o)) * silu(Wg h))              every head normed by itself, no weight

Everything between the projections and the output projection is float32.  The state of a request is one float32 row
[S of every head], zero at admission.  Launch sequence: one product for [Wq; Wk; Wv; Wg] with float32 output ->
rotation of q and k in place (steps whose entries have one token each: inside the recurrence) -> lightning_recurrence
-> gated_rmsnorm (silu gate, a group per head) -> output projection."""
from __future__ import annotations

from typing import Dict, Sequence

import torch

from ..kernels import ops
from ..profiler import bucket
from .base import MIXERS, POSITION_ENCODINGS, Mixer, ParamSpec, PartSpec, Runtime, StateSpec, build_part, register_part


@register_part(MIXERS, "retention")
class Retention(Mixer):
    graph_safe = True

    def __init__(self, runtime: Runtime, dim: int, n_heads: int, head_dim: int, v_dim: int, decay: Sequence[float],
                 position: PartSpec, eps: float):
        if n_heads <= 0 or not 0 < head_dim <= 256 or v_dim <= 0:
            raise ValueError(f"the recurrence kernel takes key sizes up to 256, got {head_dim}")
        if len(decay) != n_heads:
            raise ValueError(f"{n_heads} heads need {n_heads} decay factors, got {len(decay)}")
        self.runtime = runtime
        self.dim, self.n_heads, self.head_dim, self.v_dim = int(dim), int(n_heads), int(head_dim), int(v_dim)
        self.eps = float(eps)
        self.position = build_part(POSITION_ENCODINGS, position, runtime)
        self.decay = torch.tensor([float(x) for x in decay], dtype=torch.float32, device=runtime.device)

    def param_specs(self) -> Dict[str, ParamSpec]:
        qk, v = self.n_heads * self.head_dim, self.n_heads * self.v_dim
        return {"q": ParamSpec((qk, self.dim)), "k": ParamSpec((qk, self.dim)), "v": ParamSpec((v, self.dim)),
                "g": ParamSpec((v, self.dim)), "o": ParamSpec((self.dim, v))}

    def bind(self, params):
        if torch.device(self.runtime.device).type == "cuda":
            ops.require("state_mixers")           # the kernels of csrc/state_mixers.cu
        self.w_in = torch.cat([params[n] for n in ("q", "k", "v", "g")], dim=0).contiguous()
        self.wo = params["o"].contiguous()

    def state_spec(self) -> StateSpec:
        return StateSpec((self.n_heads * self.v_dim * self.head_dim,), torch.float32)

    def forward(self, x, ctx, cache):
        H, dk, dv = self.n_heads, self.head_dim, self.v_dim
        k_off, v_off, g_off = H * dk, 2 * H * dk, 2 * H * dk + H * dv
        with bucket("retention.in_proj"):
            proj = ops.linear(x, self.w_in, out_dtype=torch.float32)
        pos = self.position
        rot = getattr(pos, "rotary_dim", 0)
        inside = rot > 0 and ctx.max_q_len == 1 and not pos.interleaved and pos.magnitude == 1.0
        if rot and not inside:
            with bucket("retention.rope"):        # the heads of q and of k in one launch: they lie side by side
                pos.apply(proj[:, :v_off].unflatten(1, (2 * H, dk)), None, ctx)
        with bucket("retention.recurrence"):
            o = ops.lightning_recurrence(proj, 0, k_off, v_off, self.decay, cache.state, ctx, H, dk, dv, activation=None,
                                         k_scale=dk ** -0.5, inv_freq=pos.inv_freq if inside else None,
                                         rotary_dim=rot if inside else 0)
        with bucket("retention.out_norm"):
            y = ops.gated_rmsnorm(o, proj[:, g_off:g_off + H * dv], None, self.eps, H, dv, x.dtype)
        with bucket("retention.o_proj"):
            return ops.linear(y, self.wo)
