"""State space recurrence with one decay per head (Mamba-2): a [state x value] matrix per head whose decay, input and
read-out vectors depend on the token.

With h the token's normed input, H heads of ``v_dim`` values (inner = H v_dim), G groups, N = ``n_state`` and ``taps``:

    [z: inner | x: inner | B: G N | C: G N | dt: H] = W_in h
    x, B, C <- silu(conv([x | B | C]) + conv_bias)        causal, per channel, ``taps`` long, the last tap is the token's own
    dt <- softplus(dt + dt_bias)
    per head (group h // (H / G)):  S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x
    out = W_o (norm(y * silu(z)) * w)                     ``norm_groups`` equal parts, each by its own root mean square

Everything between the projections is float32.  The state of a request is one float32 row [S of every head | the
convolution's last taps-1 inputs], zero at admission.  Launch sequence: in-projection (float32 out) -> scan_conv ->
state_space -> gated_rmsnorm (gate before the norm) -> output projection.  ``pre_projection`` is everything before the
output projection."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops
from ..profiler import bucket
from .base import MIXERS, Mixer, ParamSpec, Runtime, StateSpec, register_part


@register_part(MIXERS, "state_space")
class StateSpace(Mixer):
    graph_safe = True

    def __init__(self, runtime: Runtime, dim: int, n_heads: int, v_dim: int, n_state: int, n_groups: int, taps: int,
                 norm_groups: int, eps: float):
        if not 0 < n_state <= 256 or n_heads <= 0 or v_dim <= 0 or taps < 1:
            raise ValueError(f"the state space kernel takes up to 256 states per head, got {n_state}")
        if n_groups <= 0 or n_heads % n_groups or norm_groups <= 0 or (n_heads * v_dim) % norm_groups:
            raise ValueError(f"{n_heads} heads of {v_dim} do not divide into {n_groups} groups and {norm_groups} norm groups")
        self.runtime = runtime
        self.dim, self.n_heads, self.v_dim, self.n_state = int(dim), int(n_heads), int(v_dim), int(n_state)
        self.n_groups, self.taps, self.norm_groups, self.eps = int(n_groups), int(taps), int(norm_groups), float(eps)
        self.inner = self.n_heads * self.v_dim
        self.channels = self.inner + 2 * self.n_groups * self.n_state
        self.tail_off = self.inner * self.n_state

    def param_specs(self) -> Dict[str, ParamSpec]:
        I, C, H = self.inner, self.channels, self.n_heads
        return {"in": ParamSpec((I + C + H, self.dim)), "conv": ParamSpec((C, self.taps)),
                "conv_bias": ParamSpec((C,), role="vector"), "dt_bias": ParamSpec((H,), role="vector"),
                "A_log": ParamSpec((H,), role="vector"), "D": ParamSpec((H,), role="vector", init="ones_normal"),
                "norm": ParamSpec((I,), role="vector", init="ones_normal"), "o": ParamSpec((self.dim, I))}

    def bind(self, params):
        if torch.device(self.runtime.device).type == "cuda":
            ops.require("state_mixers", "gated_states")       # the convolution and the recurrence
        f32 = lambda t: t.to(torch.float32).contiguous()
        self.w_in, self.wo = params["in"].contiguous(), params["o"].contiguous()
        self.conv, self.conv_bias = f32(params["conv"]), f32(params["conv_bias"])
        self.dt_bias, self.skip, self.norm = f32(params["dt_bias"]), f32(params["D"]), f32(params["norm"])
        self.rate = torch.exp(f32(params["A_log"])).contiguous()

    @property
    def out_width(self) -> int:
        return self.inner

    def state_spec(self) -> StateSpec:
        size = self.tail_off + (self.taps - 1) * self.channels
        return StateSpec((-(-size // 4) * 4,), torch.float32)        # rows start on 16-byte boundaries

    def forward(self, x, ctx, cache):
        y = self.pre_projection(x, ctx, cache)
        with bucket("state_space.o_proj"):
            return ops.linear(y, self.wo)

    def pre_projection(self, x, ctx, cache, out=None, out_scale: float = 1.0):
        """The normed rows [n, inner] in the run dtype, times ``out_scale``; written into ``out`` (a view of columns of
        wider rows) when given."""
        I, C = self.inner, self.channels
        with bucket("state_space.in_proj"):
            proj = ops.linear(x, self.w_in, out_dtype=torch.float32)
        xbc, dt = proj[:, I:I + C], proj[:, I + C:]
        with bucket("state_space.conv"):
            conv, _ = ops.scan_conv(xbc, self.conv, self.conv_bias, cache.state, self.tail_off, ctx, C, self.taps)
        with bucket("state_space.recurrence"):
            y = ops.state_space(conv, xbc, dt, self.dt_bias, self.rate, self.skip, cache.state, self.tail_off, ctx,
                                self.n_heads, self.n_groups, self.n_state, self.v_dim, self.taps)
        with bucket("state_space.out_norm"):
            return ops.gated_rmsnorm(y, proj[:, :I], self.norm, self.eps, self.norm_groups, I // self.norm_groups, x.dtype,
                                     gate_first=True, out=out, out_scale=out_scale)
