"""Mamusun as a ModelSpec.

Token embedding without positions of its own; per layer the `post_norm` arrangement (a norm after the sum of the stream,
times the configuration's alpha, and a sublayer's output) with RMS norms whose gains are stored around zero, and after
the layer a weighted sum over depth (`depth_average`).  A layer's mixer is a windowed attention with a norm a head and no
rotation, which may read the keys and values that an earlier layer cached; an attention over all keys whose values
are its keys as projected, with biases, norms over whole rows, a rotation with YaRN and a learned sink; or two members
side by side: a windowed attention whose heads are rotated in part, in neighbouring pairs, with frequencies scaled by
bands of wavelengths, and normed after the rotation, and Griffin's recurrent block; each member's output is RMS-normed
with a gain of its own and the two are added with a half each.  The feed-forward is dense with PolyNorm, or experts of the
clamped gated form chosen by a router with a bias and weighed by a softmax over the chosen, or absent.  A last norm, an
untied head.

The design's fixed numbers stand here: 1.702 and the + 1 of the clamped gate, the half and half of the two members, and
the factor 8 on the recurrence's decays; everything else comes from the configuration.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.mamusun import MamusunConfig
from ..parts.spec import Application, LayerSpec, ModelSpec, PartSpec

GATE_ALPHA = 1.702
UP_SHIFT = 1.0
MEMBER_FACTOR = 0.5
DECAY_FACTOR = 8.0


def _heads(d: int, m: dict, eps: float) -> dict:
    return {"width": d, "n_heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
            "scale": m["scale"], "qkv": ("q", "k", "v"), "out": "o", "stored": "out_in", "bias": False, "suffix": "",
            "norm_eps": eps}


def build_spec(cfg: MamusunConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("rmsnorm", name, {"width": d, "eps": eps, "weight": "", "offset": 1.0})  # noqa: E731
    layers, schedule, ignored = [], [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer["mixer"]
        cache_of = None
        if layer["type"] == "attention":
            cache_of = m.get("kv_from")
            mixer = PartSpec("causal_attention", p + "mix.", {
                **_heads(d, m, eps), "window": m["mask"]["size"], "qk_norm": ("q.norm", "k.norm"), "qk_norm_scope": "head",
                "shares_cache": cache_of is not None})
        elif layer["type"] == "attention_2":
            rot = m["rot"]
            mixer = PartSpec("causal_attention", p + "mix.", {
                **_heads(d, m, eps), "qkv_bias": ".b", "values_are_keys": True, "qk_norm": ("q.norm", "k.norm"),
                "rotary": (rot["dims"], rot["base"], False, rot.get("scaling")), "sink": "sink"})
        else:
            a, r = m["left"], m["right"]
            rot = a["rot"]
            scaling = None if rot.get("scaling") is None else {"kind": "bands", **rot["scaling"]}
            left = PartSpec("causal_attention", p + "mix.left.", {
                **_heads(d, a, eps), "window": a["mask"]["size"], "rotary": (rot["dims"], rot["base"], True, scaling), "unit_qk": True})
            right = PartSpec("rglru", p + "mix.right.", {"width": d, "inner": r["width"], "blocks": r["blocks"], "conv": r["conv"],
                                                         "factor": DECAY_FACTOR})
            mixer = PartSpec("parallel", p + "mix.", {
                "width": d, "members": (("left", left, MEMBER_FACTOR), ("right", right, MEMBER_FACTOR)),
                "out_norms": ("left.out", "right.out"), "eps": eps})
        mlp = layer.get("mlp")
        if mlp is None:
            ffn = None
            ignored.append(rf"l{i}\.norm2")
        elif mlp["kind"] == "dense":
            ffn = PartSpec("dense", p + "mlp.", {
                "width": d, "inner": mlp["ff"], "activation": "poly_norm", "act": "act", "act_eps": eps, "up": "up", "down": "down",
                "stored": "out_in", "bias": False, "suffix": "", "any_size": True})
        else:
            ffn = PartSpec("routed_experts", p + "mlp.", {
                "width": d, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "inner": mlp["expert"]["ff"],
                "limit": mlp["expert"]["limit"], "alpha": GATE_ALPHA, "shift": UP_SHIFT, "scores": "softmax",
                "correction": "router.b"})
        schedule.append(Application(i, cache_of))
        layers.append(LayerSpec("post_norm", norm(p + "norm1"), mixer, norm(p + "norm2") if ffn is not None else None, ffn,
                                addons=(PartSpec("depth_average", p, {"layers": i + 1}),), block_params={"alpha": cfg.alpha}))
    return ModelSpec(width=d, vocab_size=cfg.vocab, token_table="embed", position=PartSpec("none", ""),
                     layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"), head="head",
                     ignored_tensors=tuple(ignored))


register_architecture(MamusunConfig.architecture, MamusunConfig, build_spec)
