"""Matrix memory (the mLSTM of xLSTM): a [key x value] matrix and a key vector per head with exponential gates.

With h the token's normed input and H heads:

    q = Wq h / sqrt(dim),  k = Wk h  (H x dim),   v = Wv h  (H x v_dim)
    i = c tanh((Wi h + bi) / c),   f = logsigmoid(c tanh((Wf h + bf) / c))        per head, c = ``gate_cap``
    m_t = max(f + m_(t-1), i)      from 0
    S <- exp(f + m_(t-1) - m_t) S + exp(i - m_t) k v^T,   n likewise with k alone;   both from 0
    o = S^T q / (max(|n . q|, exp(-m_t)) + 1e-6)
    out = Wo (concat_heads(o / rms(o)) * w * sigmoid(Wg h))                       every head normed by itself

Everything between the projections is float32.  The state of a request is one float32 row [S and n of every head | the
running maximum of every head], zero at admission.  Launch sequence: one product for [Wq; Wk; Wv; Wg; Wi; Wf] with float32
output -> matrix_memory -> gated_rmsnorm (a group per head, divides by the denominator first) -> output projection.
``pre_projection`` is everything before the output projection."""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops
from ..profiler import bucket
from .base import MIXERS, Mixer, ParamSpec, Runtime, StateSpec, register_part


@register_part(MIXERS, "matrix_memory")
class MatrixMemory(Mixer):
    graph_safe = True

    def __init__(self, runtime: Runtime, dim: int, n_heads: int, head_dim: int, v_dim: int, gate_cap: float, eps: float):
        if n_heads <= 0 or not 0 < head_dim <= 256 or v_dim <= 0:
            raise ValueError(f"the matrix memory kernel takes key sizes up to 256, got {head_dim}")
        if not gate_cap > 0:
            raise ValueError(f"the gates' cap must be positive, got {gate_cap}")
        self.runtime = runtime
        self.dim, self.n_heads, self.head_dim, self.v_dim = int(dim), int(n_heads), int(head_dim), int(v_dim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.m_off = self.n_heads * (self.v_dim + 1) * self.head_dim

    def param_specs(self) -> Dict[str, ParamSpec]:
        qk, v, H = self.n_heads * self.head_dim, self.n_heads * self.v_dim, self.n_heads
        return {"q": ParamSpec((qk, self.dim)), "k": ParamSpec((qk, self.dim)), "v": ParamSpec((v, self.dim)),
                "g": ParamSpec((v, self.dim)), "i": ParamSpec((H, self.dim)), "f": ParamSpec((H, self.dim)),
                "i_bias": ParamSpec((H,), role="vector"), "f_bias": ParamSpec((H,), role="vector"),
                "norm": ParamSpec((v,), role="vector", init="ones_normal"), "o": ParamSpec((self.dim, v))}

    def bind(self, params):
        if torch.device(self.runtime.device).type == "cuda":
            ops.require("gated_states")
        f32 = lambda t: t.to(torch.float32).contiguous()
        self.w_in = torch.cat([params[n] for n in ("q", "k", "v", "g", "i", "f")], dim=0).contiguous()
        self.i_bias, self.f_bias, self.norm = f32(params["i_bias"]), f32(params["f_bias"]), f32(params["norm"])
        self.wo = params["o"].contiguous()

    @property
    def out_width(self) -> int:
        return self.n_heads * self.v_dim

    def state_spec(self) -> StateSpec:
        size = self.m_off + ops.MATRIX_MEMORY_RECORD * self.n_heads
        return StateSpec((-(-size // 4) * 4,), torch.float32)        # rows start on 16-byte boundaries

    def forward(self, x, ctx, cache):
        y = self.pre_projection(x, ctx, cache)
        with bucket("matrix_memory.o_proj"):
            return ops.linear(y, self.wo)

    def pre_projection(self, x, ctx, cache, out=None, out_scale: float = 1.0):
        """The normed and gated heads [n, H v_dim] in the run dtype, times ``out_scale``; written into ``out`` (a view of
        columns of wider rows) when given."""
        H, dk, dv = self.n_heads, self.head_dim, self.v_dim
        k_off, v_off = H * dk, 2 * H * dk
        g_off = v_off + H * dv
        i_off = g_off + H * dv
        with bucket("matrix_memory.in_proj"):
            proj = ops.linear(x, self.w_in, out_dtype=torch.float32)
        with bucket("matrix_memory.recurrence"):
            o, den = ops.matrix_memory(proj, 0, k_off, v_off, i_off, i_off + H, self.i_bias, self.f_bias, self.gate_cap,
                                       dk ** -0.5, cache.state, self.m_off, ctx, H, dk, dv)
        with bucket("matrix_memory.out_norm"):
            return ops.gated_rmsnorm(o, proj[:, g_off:g_off + H * dv], self.norm, self.eps, H, dv, x.dtype,
                                     gate_act="sigmoid", den=den, out=out, out_scale=out_scale)
