"""A plain, slow implementation of the Guvolix design in float64 on the CPU: whole sequences, one function per
mechanism, python loops where the definition is a recurrence.  It shares no code with the package; the tests compare
the engine with it.

Notation: h is a [T, d] matrix of one sequence's rows, W x means ``x @ W.T`` for a weight stored [out, in]."""
from __future__ import annotations

import json
import math
from pathlib import Path
from typing import Dict, Optional, Sequence

import torch

F = torch.float64


def f64(t):
    return t.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rms_unit(x, eps: float):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps: float):
    return rms_unit(x, eps) * f64(w)


# ---------------------------------------------------------------------------------------------- attention
def angle_rates(rot: dict):
    """One rate per pair i < dims/2: base^(-2i/dims), divided by a factor, or (with an ``original`` length) divided for
    the long waves only, with a ramp between."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc and "original" in sc:
            wave, n = 2.0 * math.pi / f, sc["original"]
            if wave > n / sc["low"]:
                f = f / sc["factor"]
            elif wave >= n / sc["high"]:
                s = (n / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        elif sc:
            f = f / sc["factor"]
        out.append(f)
    return out


def rotate_halves(x, rot: dict):
    """x [T, heads, D]: number i and number i + dims/2 of a head, i < dims/2, turn by position * rate_i."""
    T, half = x.shape[0], rot["dims"] // 2
    out = x.clone()
    for i, f in enumerate(angle_rates(rot)):
        a = torch.arange(T, dtype=F) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def visible(T: int, window: Optional[int], keep: int = 0):
    """[T, T]: query i sees key j <= i inside its window, or among the first ``keep`` of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if window:
        see = see & ((i - j < window) | (j < keep))
    return see


def attend(q, k, v, scale: float, window: Optional[int] = None, keep: int = 0, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; exp(sink_h) joins the denominator only."""
    T, H, _ = q.shape
    G = k.shape[1]
    see = visible(T, window, keep)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~see, float("-inf"))
        m = s.amax(dim=1, keepdim=True)
        e = torch.exp(s - m)
        den = e.sum(dim=1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(f64(sink)[h] - m)
        out[:, h] = (e / den) @ v[:, g]
    return out


def gated_attention(h, w, m: dict):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ f64(w["q"]).T).view(T, H, m["dim"])
    k = (h @ f64(w["k"]).T).view(T, G, m["dim"])
    v = (h @ f64(w["v"]).T).view(T, G, m["vdim"])
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"])
    mask = m.get("mask") or {}
    o = attend(q, k, v, m["scale"], mask.get("size"), mask.get("keep_first", 0), w["sink"]).reshape(T, -1)
    return (o * torch.sigmoid(h @ f64(w["g"]).T)) @ f64(w["o"]).T


# ---------------------------------------------------------------------------------------------- recurrences
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] (the last one is the current token's), zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    out = f64(bias).expand(T, C).clone()
    for t in range(T):
        for j in range(n):
            if t - (n - 1 - j) >= 0:
                out[t] += f64(taps)[:, j] * x[t - (n - 1 - j)]
    return out


def scalar_decay_state(x, B, C, dt, a_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H]: per head S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    out = torch.zeros(T, H, V, dtype=F)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, V, dtype=F)
        rate = math.exp(float(a_log[h]))
        for t in range(T):
            S = math.exp(-rate * float(dt[t, h])) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S.T @ C[t, g] + float(D[h]) * x[t, h]
    return out


def grouped_gated_norm(y, z, w, groups: int, eps: float):
    """y silu(z), each of ``groups`` equal parts divided by its own root mean square, times w."""
    T, n = y.shape
    u = (y * silu(z)).view(T, groups, n // groups)
    return rms_unit(u, eps).reshape(T, n) * f64(w)


def state_space_dual(h, w, m: dict, eps: float):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    zxbcdt = h @ f64(w["in"]).T
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner:2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + f64(w["dt_bias"]))
    y = scalar_decay_state(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, f64(w["A_log"]), f64(w["D"]))
    return grouped_gated_norm(y.reshape(T, inner), z, w["norm"], m["norm_groups"], eps) @ f64(w["o"]).T


def matrix_memory(q, k, v, i_log, f_log):
    """q, k [T, H, D], v [T, H, V], log gates [T, H]: the running maximum starts at 0."""
    T, H, D = q.shape
    V = v.shape[2]
    out = torch.zeros(T, H, V, dtype=F)
    for h in range(H):
        S, n, m = torch.zeros(D, V, dtype=F), torch.zeros(D, dtype=F), 0.0
        for t in range(T):
            i, f = float(i_log[t, h]), float(f_log[t, h])
            m_new = max(f + m, i)
            a, b = math.exp(f + m - m_new), math.exp(i - m_new)
            S = a * S + b * torch.outer(k[t, h], v[t, h])
            n = a * n + b * k[t, h]
            m = m_new
            out[t, h] = (S.T @ q[t, h]) / (max(abs(float(n @ q[t, h])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, w, mx: dict, eps: float):
    T, H, D, V, cap = h.shape[0], mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    q = (h @ f64(w["q"]).T).view(T, H, D) * D ** -0.5
    k = (h @ f64(w["k"]).T).view(T, H, D)
    v = (h @ f64(w["v"]).T).view(T, H, V)
    i_log = cap * torch.tanh((h @ f64(w["i"]).T + f64(w["i.b"])) / cap)
    f_log = -softplus(-cap * torch.tanh((h @ f64(w["f"]).T + f64(w["f.b"])) / cap))
    o = rms_unit(matrix_memory(q, k, v, i_log, f_log), eps).reshape(T, H * V)
    return (o * f64(w["norm"]) * torch.sigmoid(h @ f64(w["g"]).T)) @ f64(w["o"]).T


# ---------------------------------------------------------------------------------------------- mixers
def _side(w, side: str):
    return {k[len(side) + 1:]: v for k, v in w.items() if k.startswith(side + ".")}


def mix_normed(h, w, m: dict, eps: float):
    """Attention beside the state space recurrence: half the sum of the outputs, each normed over the width."""
    wl, wr = _side(w, "left"), _side(w, "right")
    left = rms_norm(gated_attention(h, wl, m["left"]), wl["out"], eps)
    right = rms_norm(state_space_dual(h, wr, m["right"], eps), wr["out"], eps)
    return 0.5 * (left + right)


def mix_scaled(h, w, m: dict, eps: float):
    """Attention beside the matrix memory: a weighted sum with two constants."""
    return (m["left_scale"] * gated_attention(h, _side(w, "left"), m["left"])
            + m["right_scale"] * mlstm(h, _side(w, "right"), m["right"], eps))


# ---------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h, w):
    return gelu(h @ f64(w["up"]).T) @ f64(w["down"]).T


def gated_ff(h, gate, up, down):
    return (silu(h @ f64(gate).T) * (h @ f64(up).T)) @ f64(down).T


def route(h, router, correction, top: int):
    """(numbers [T, top], weights [T, top]): softmax scores, chosen by score plus correction, weighted by the chosen
    scores over their sum."""
    s = torch.softmax(h @ f64(router).T, dim=-1)
    ids = torch.argsort(s + f64(correction), dim=-1, descending=True, stable=True)[:, :top]
    chosen = s.gather(1, ids)
    return ids, chosen / (chosen.sum(dim=-1, keepdim=True) + 1e-20)


def routed_ff(h, w, f: dict):
    r = f["router"]
    ids, wts = route(h, w["router"], w["correction"], r["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for c, e in enumerate(ids[t].tolist()):
            row = h[t:t + 1]
            out = row if e >= r["experts"] else gated_ff(row, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
            y[t] += wts[t, c] * out[0]
    if f.get("shared") is not None:
        y = y + torch.sigmoid(h @ f64(w["shared.sg"]).T) * gated_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return y


# ---------------------------------------------------------------------------------------------- the model
def layer_forward(x, cfg: dict, tensors: Dict[str, torch.Tensor], i: int):
    layer, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    sub = lambda name: {k[len(p + name) + 1:]: v for k, v in tensors.items() if k.startswith(p + name + ".")}
    h = rms_norm(x, tensors[p + "norm1"], eps)
    mix = {"parallel": mix_normed, "parallel_2": mix_scaled}[layer["type"]]
    y = mix(h, sub("mix"), layer["mixer"], eps)
    f = layer.get("mlp")
    if f is not None:
        y = y + (dense_ff(h, sub("mlp")) if f["kind"] == "dense" else routed_ff(h, sub("mlp"), f))
    return x + y


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: Sequence[int], return_layers: bool = False):
    """float64 logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    x = f64(tensors["embed"])[list(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, cfg, tensors, i)
        after.append(x)
    logits = rms_norm(x, tensors["final.norm"], cfg["norm"]["eps"]) @ f64(tensors["head"]).T
    return (logits, torch.stack(after)) if return_layers else logits


# ---------------------------------------------------------------------------------------------- a model folder
def read_tensors(path) -> Dict[str, torch.Tensor]:
    """All tensors of a safetensors file by name; bfloat16 comes back as float32 with the same values."""
    import struct
    import numpy as np
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    out = {}
    for name, meta in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = (8 + n + o for o in meta["data_offsets"])
        if meta["dtype"] == "BF16":
            arr = (np.frombuffer(raw[lo:hi], dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(raw[lo:hi], dtype={"F32": np.float32, "I32": np.int32}[meta["dtype"]]).copy()
        out[name] = torch.from_numpy(arr).reshape(meta["shape"])
    return out


def read_model_folder(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_tensors(folder / "model.safetensors")
