"""A plain, slow implementation of the Podizen design in float64 on the CPU: whole sequences, one function per
mechanism, python loops where the definition is a recurrence.  It shares no code with the package; the tests compare
the engine with it.

Notation: h is a [T, d] matrix of one sequence's rows, W x means ``x @ W.T`` for a weight stored [out, in]."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, List, Optional, Sequence

import torch

F = torch.float64


def f64(t):
    return t.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def rms_unit(x, eps: float):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps: float):
    return rms_unit(x, eps) * f64(w)


def rotate_halves(x, base: float, dims: int):
    """x [T, heads, D]: number i and number i + dims/2 of a head, i < dims/2, turn by position * base^(-2i/dims)."""
    T, half = x.shape[0], dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(T, dtype=F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def bias_slopes(heads: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def pooled_blocks(x, pool: int):
    """x [T, G, D] -> the means of its whole blocks of ``pool`` rows, [T // pool, G, D]."""
    n = x.shape[0] // pool
    return torch.stack([x[b * pool:(b + 1) * pool].mean(dim=0) for b in range(n)]) if n else x[:0]


def attend(q, k, v, scale: float, window: Optional[int] = None, pool: Optional[int] = None,
           slopes: Optional[Sequence[float]] = None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V].  Position i sees the tokens j <= i with i - j < window (all
    of them without a window); with ``pool`` P also one mean key and value for every block of P tokens whose last token
    is at most i - window.  ``slopes``: slope_h * (i - j) is taken off the scaled score of a token."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if window:
        see = see & (i - j < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        keys, values, seen = k[:, g], v[:, g], see
        s = (q[:, h] @ keys.T) * scale
        if slopes is not None:
            s = s - slopes[h] * (i - j).to(F)
        if pool:
            pk, pv = pooled_blocks(k, pool)[:, g], pooled_blocks(v, pool)[:, g]
            last = torch.arange(pk.shape[0])[None, :] * pool + pool - 1
            s = torch.cat([s, (q[:, h] @ pk.T) * scale], dim=1)
            seen = torch.cat([see, last <= i - window], dim=1)
            values = torch.cat([values, pv], dim=0)
        p = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=1)
        out[:, h] = p @ values
    return out


def biased_attention(h, w, m: dict):
    """Grouped-query attention with a distance bias, a sliding window and an output gate; no rotation."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ f64(w["q"]).T).view(T, H, m["dim"])
    k = (h @ f64(w["k"]).T).view(T, G, m["dim"])
    v = (h @ f64(w["v"]).T).view(T, G, m["vdim"])
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), slopes=bias_slopes(H)).reshape(T, -1)
    return (o * torch.sigmoid(h @ f64(w["g"]).T)) @ f64(w["o"]).T


def pooled_attention(h, w, m: dict, eps: float):
    """Grouped-query attention with weighted head norms, then rotation, and a window with pooled blocks before it."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm((h @ f64(w["q"]).T).view(T, H, m["dim"]), w["q.norm"], eps)
    k = rms_norm((h @ f64(w["k"]).T).view(T, G, m["dim"]), w["k.norm"], eps)
    v = (h @ f64(w["v"]).T).view(T, G, m["vdim"])
    q, k = (rotate_halves(t, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    mask = m.get("mask") or {}
    o = attend(q, k, v, m["scale"], mask.get("size"), mask.get("pool"))
    return o.reshape(T, -1) @ f64(w["o"]).T


def decaying_state(q, k, v, decay: Sequence[float]):
    """q, k [T, H, D], v [T, H, V]: per head S <- decay_h S + k v^T from zero, o = S^T q."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for j in range(H):
        S = torch.zeros(D, v.shape[2], dtype=F)
        for t in range(T):
            S = decay[j] * S + torch.outer(k[t, j], v[t, j])
            out[t, j] = S.T @ q[t, j]
    return out


def retention(h, w, m: dict, eps: float):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    q = (h @ f64(w["q"]).T).view(T, H, D)
    k = (h @ f64(w["k"]).T).view(T, H, D)
    v = (h @ f64(w["v"]).T).view(T, H, m["vdim"])
    q, k = (rotate_halves(t, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    o = rms_unit(decaying_state(q, k * D ** -0.5, v, m["decay"]), eps).reshape(T, -1)
    return (o * silu(h @ f64(w["g"]).T)) @ f64(w["o"]).T


def parallel_mixer(h, w, m: dict, eps: float):
    """Half the sum of the two mixers' outputs, each RMS-normed over the width first."""
    part = lambda side: {k[len(side) + 1:]: v for k, v in w.items() if k.startswith(side + ".")}
    wl, wr = part("left"), part("right")
    left = rms_norm(pooled_attention(h, wl, m["left"], eps), wl["out"], eps)
    right = rms_norm(retention(h, wr, m["right"], eps), wr["out"], eps)
    return 0.5 * (left + right)


def gated_ff(h, gate, up, down):
    return (silu(h @ f64(gate).T) * (h @ f64(up).T)) @ f64(down).T


def route(h, router, top: int, groups: int, keep: int):
    """(expert numbers [T, top], weights [T, top]): softmax over all experts; only the experts of the ``keep`` groups
    of neighbours with the largest scores take part; weights are the chosen scores over their sum."""
    s = torch.softmax(h @ f64(router).T, dim=-1)
    T, E = s.shape
    per = E // groups
    ids, wts = torch.zeros(T, top, dtype=torch.int64), torch.zeros(T, top, dtype=F)
    for t in range(T):
        score = s[t].view(groups, per).amax(dim=1)
        kept = set(torch.argsort(score, descending=True, stable=True)[:keep].tolist())
        order = [e for e in torch.argsort(s[t], descending=True, stable=True).tolist() if e // per in kept]
        ids[t] = torch.tensor(order[:top])
        wts[t] = s[t, ids[t]] / (s[t, ids[t]].sum() + 1e-20)
    return ids, wts


def routed_ff(h, w, f: dict):
    r = f["router"]
    g = r.get("groups") or {}
    ids, wts = route(h, w["router"], r["top"], g.get("count", 1), g.get("keep", 1))
    rows = []
    for t in range(h.shape[0]):
        y = sum(wts[t, c] * gated_ff(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
                for c, e in enumerate(ids[t].tolist()))
        rows.append(y)
    y = torch.cat(rows)
    if f.get("shared") is not None:
        y = y + gated_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return y


def layer_forward(x, cfg: dict, tensors: Dict[str, torch.Tensor], i: int):
    """The layer's own result, before the averaging over depth."""
    layer, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    sub = lambda name: {k[len(p + name) + 1:]: v for k, v in tensors.items() if k.startswith(p + name + ".")}
    h, m = rms_norm(x, tensors[p + "norm1"], eps), layer["mixer"]
    if layer["type"] == "attention":
        y = biased_attention(h, sub("mix"), m)
    elif layer["type"] == "parallel":
        y = parallel_mixer(h, sub("mix"), m, eps)
    else:
        raise ValueError(layer["type"])
    x = x + rms_norm(y, tensors[p + "norm1b"], eps)
    f = layer.get("mlp")
    if f is not None:
        y = routed_ff(rms_norm(x, tensors[p + "norm2"], eps), sub("mlp"), f)
        x = x + rms_norm(y, tensors[p + "norm2b"], eps)
    return x


def depth_average(states: List[torch.Tensor], weights):
    return sum(float(wj) * s for wj, s in zip(f64(weights), states))


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: Sequence[int], return_layers: bool = False):
    """float64 logits [T, vocab] of one whole sequence (and the residual stream that goes on after every layer)."""
    x = f64(tensors["embed"])[list(tokens)]
    states, after = [x], []
    for i in range(len(cfg["layers"])):
        states.append(layer_forward(x, cfg, tensors, i))
        x = depth_average(states, tensors[f"l{i}.dwa"])
        after.append(x)
    logits = rms_norm(x, tensors["final.norm"], cfg["norm"]["eps"]) @ f64(tensors["embed"]).T
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
