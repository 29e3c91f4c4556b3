"""The Guvolix design as a model description: the embedding times a constant; layers of one norm whose mixer and
feed-forward both read it and join the residual together; every mixer is a gated sliding-window attention (first tokens
that stay visible, a learned softmax sink, scaled rotary frequencies) side by side with a recurrence, either a state space
one with a scalar decay per head, both outputs normed over the width and halved, or a matrix memory, both outputs scaled
by constants; a feed-forward that is two matrices around an exact gelu, or routed silu-gated experts with identity experts
and a gated shared one, or absent; a final norm and an untied head.

Checkpoint names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.left.{q, k, v, sink, g, o}``, ``l<i>.mix.right.{in, conv, conv.b,
dt_bias, A_log, D, norm, o}`` and ``l<i>.mix.{left, right}.out``, or ``l<i>.mix.right.{q, k, v, g, i, i.b, f, f.b, norm,
o}``, ``l<i>.mlp.{up, down}`` or ``l<i>.mlp.{router, correction, e<j>.gate, e<j>.up, e<j>.down, shared.gate, shared.up,
shared.down, shared.sg}``, ``final.norm``, ``head``."""
from __future__ import annotations

from ..config.guvolix_config import GuvolixConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, RunEntry

_STATE_SPACE_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
                      "norm": "norm", "o": "o"}
_MATRIX_MEMORY_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "i": "i", "f": "f", "i_bias": "i.b", "f_bias": "f.b",
                        "norm": "norm", "o": "o"}


def _position(m: dict) -> PartSpec:
    rot = m.get("rot")
    if not rot or not rot["dims"]:
        return PartSpec("none")
    scaling = rot.get("scaling") or None
    if scaling and "original" in scaling:
        scaling = dict(rope_type="llama3", factor=scaling["factor"], low_freq_factor=scaling["low"],
                       high_freq_factor=scaling["high"], original_max_position_embeddings=scaling["original"])
    elif scaling:
        scaling = dict(rope_type="linear", factor=scaling["factor"])
    return PartSpec("rope", dict(head_dim=m["dim"], theta=rot["base"], scaling=scaling, rotary_dim=rot["dims"],
                                 interleaved=False))


def build_guvolix(cfg: GuvolixConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = PartSpec("rmsnorm", dict(dim=d, eps=eps, single_rounding=True))
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        a, b = m["left"], m["right"]
        mask = a.get("mask") or {}
        left = PartSpec("sink_attention", dict(
            dim=d, n_heads=a["heads"], n_kv_heads=a["kv_heads"], head_dim=a["dim"], v_dim=a["vdim"], scale=a["scale"],
            position=_position(a), window=mask.get("size"), keep_first=mask.get("keep_first"), sink=True, gate=True))
        names = {"norm1.weight": p + "norm1"}
        names.update({f"mixer.left.{k}": p + "mix.left." + k for k in ("q", "k", "v", "sink", "g", "o")})
        if layer["type"] == "parallel":
            right = PartSpec("state_space", dict(dim=d, n_heads=b["heads"], v_dim=b["vdim"], n_state=b["state"],
                                                 n_groups=b["groups"], taps=b["conv"], norm_groups=b["norm_groups"], eps=eps))
            mixer = PartSpec("parallel", dict(left=left, right=right, left_scale=0.5, right_scale=0.5, out_norm_eps=eps))
            right_names = _STATE_SPACE_NAMES
            names.update({f"mixer.{side}_out": f"{p}mix.{side}.out" for side in ("left", "right")})
        else:
            right = PartSpec("matrix_memory", dict(dim=d, n_heads=b["heads"], head_dim=b["dim"], v_dim=b["vdim"],
                                                   gate_cap=b["gate_cap"], eps=eps))
            mixer = PartSpec("parallel", dict(left=left, right=right, left_scale=m["left_scale"],
                                              right_scale=m["right_scale"]))
            right_names = _MATRIX_MEMORY_NAMES
        names.update({f"mixer.right.{k}": p + "mix.right." + v for k, v in right_names.items()})
        f = layer.get("mlp")
        if f is None:
            layers.append(LayerSpec({"norm1": norm, "mixer": mixer}, names, "parallel_prenorm_mixer"))
            continue
        if f["kind"] == "dense":
            ffn = PartSpec("mlp", dict(dim=d, intermediate=f["ff"], activation="gelu"))
            names.update({f"ffn.{k}": p + "mlp." + k for k in ("up", "down")})
        else:
            r, shared = f["router"], (f.get("shared") or {}).get("ff", 0)
            ffn = PartSpec("routed_glu", dict(dim=d, intermediate=f["expert"]["ff"], n_experts=r["experts"], top=r["top"],
                                              bias=False, scores="softmax", correction=True, identity=r.get("identity", 0),
                                              shared=shared, shared_gate=bool(shared)))
            names.update({"ffn.router": p + "mlp.router", "ffn.correction": p + "mlp.correction"})
            for e in range(r["experts"]):
                names.update({f"ffn.{k}{e}": f"{p}mlp.e{e}.{k}" for k in ("gate", "up", "down")})
            if shared:
                names.update({f"ffn.shared.{k}": f"{p}mlp.shared.{k}" for k in ("gate", "up", "down")})
                names["ffn.shared_gate"] = p + "mlp.shared.sg"
        layers.append(LayerSpec({"norm1": norm, "mixer": mixer, "ffn": ffn}, names, "parallel_prenorm"))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden_size=d, layers=layers, order=[RunEntry(i) for i in range(len(layers))],
        final_norm=norm, embed_name="embed", final_norm_names={"weight": "final.norm"}, lm_head_name="head",
        embed_scale=cfg.embed_scale)
