"""The Podizen design as a model description: layers whose branches are RMS-normed before and after each sublayer, and
whose result is averaged with all earlier results and the embedding by learned numbers before it goes on; per layer one
of two mixers, grouped-query attention with a distance bias, a sliding window and an output gate, or, side by side and
each normed over the width, a windowed attention that also sees one mean key and value per block of tokens before its
window, and a retention; a feed-forward of routed silu-gated experts with a shared one, or none; a final norm and the
embedding table as the head.

Checkpoint names: ``embed``, ``l<i>.{norm1, norm1b, norm2, norm2b, dwa}``, ``l<i>.mix.{q, k, v, g, o}``,
``l<i>.mix.left.{q, k, v, q.norm, k.norm, o, out}``, ``l<i>.mix.right.{q, k, v, g, o, out}``,
``l<i>.mlp.{router, e<j>.gate, e<j>.up, e<j>.down, shared.gate, shared.up, shared.down}``, ``final.norm``."""
from __future__ import annotations

from ..config.podizen_config import PodizenConfig
from ..parts.base import PartSpec
from ..parts.sink_attention import geometric_slopes
from .spec import LayerSpec, ModelSpec, RunEntry


def _position(m: dict) -> PartSpec:
    rot = m.get("rot")
    if not rot or not rot["dims"]:
        return PartSpec("none")
    return PartSpec("rope", dict(head_dim=m["dim"], theta=rot["base"], scaling=None, rotary_dim=rot["dims"],
                                 interleaved=False))


def build_podizen(cfg: PodizenConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = PartSpec("rmsnorm", dict(dim=d, eps=eps, single_rounding=True))
    layers, ignore = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        names = {"norm1.weight": p + "norm1", "norm1b.weight": p + "norm1b", "average.weight": p + "dwa"}
        if layer["type"] == "attention":
            mixer = PartSpec("sink_attention", dict(
                dim=d, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"],
                scale=m["scale"], position=PartSpec("none"), window=(m.get("mask") or {}).get("size"), gate=True,
                bias_slopes=geometric_slopes(m["heads"])))
            names.update({f"mixer.{k}": p + "mix." + k for k in ("q", "k", "v", "g", "o")})
        else:
            a, b = m["left"], m["right"]
            mask = a.get("mask") or {}
            left = PartSpec("sink_attention", dict(
                dim=d, n_heads=a["heads"], n_kv_heads=a["kv_heads"], head_dim=a["dim"], v_dim=a["vdim"],
                scale=a["scale"], position=_position(a), qk_norm_eps=eps, qk_norm_weight=True, qk_norm_first=True,
                window=mask.get("size"), pool=mask.get("pool")))
            right = PartSpec("retention", dict(dim=d, n_heads=b["heads"], head_dim=b["dim"], v_dim=b["vdim"],
                                               decay=list(b["decay"]), position=_position(b), eps=eps))
            mixer = PartSpec("parallel", dict(left=left, right=right, left_scale=0.5, right_scale=0.5,
                                              out_norm_eps=eps))
            names.update({f"mixer.left.{k}": p + "mix.left." + k for k in ("q", "k", "v", "o")})
            names.update({"mixer.left.q_norm": p + "mix.left.q.norm", "mixer.left.k_norm": p + "mix.left.k.norm"})
            names.update({f"mixer.right.{k}": p + "mix.right." + k for k in ("q", "k", "v", "g", "o")})
            names.update({f"mixer.{side}_out": f"{p}mix.{side}.out" for side in ("left", "right")})
        parts = {"norm1": norm, "mixer": mixer, "norm1b": norm}
        average = PartSpec("learned", dict(count=i + 2))
        f = layer.get("mlp")
        if f is None:
            layers.append(LayerSpec({**parts, "average": average}, names, "sandwich_mixer_averaged"))
            ignore += [p + "norm2", p + "norm2b"]        # norms around no feed-forward are never applied
            continue
        r = f["router"]
        g = r.get("groups") or {}
        shared = (f.get("shared") or {}).get("ff", 0)
        ffn = PartSpec("routed_glu", dict(dim=d, intermediate=f["expert"]["ff"], n_experts=r["experts"], top=r["top"],
                                          bias=False, scores="softmax", n_groups=g.get("count", 1),
                                          keep_groups=g.get("keep", 1), shared=shared))
        names.update({"norm2.weight": p + "norm2", "norm2b.weight": p + "norm2b", "ffn.router": p + "mlp.router"})
        for e in range(r["experts"]):
            names.update({f"ffn.{k}{e}": f"{p}mlp.e{e}.{k}" for k in ("gate", "up", "down")})
        if shared:
            names.update({f"ffn.shared.{k}": f"{p}mlp.shared.{k}" for k in ("gate", "up", "down")})
        layers.append(LayerSpec({**parts, "norm2": norm, "ffn": ffn, "norm2b": norm, "average": average}, names,
                                "sandwich_averaged"))
    return ModelSpec(
        vocab_size=cfg.vocab_size, hidden_size=d, layers=layers, order=[RunEntry(i) for i in range(len(layers))],
        final_norm=norm, embed_name="embed", final_norm_names={"weight": "final.norm"}, lm_head_name=None,
        ignore_names=tuple(ignore), depth_average=True)
