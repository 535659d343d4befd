"""Podenex as a ModelSpec.

Token embedding without positions of its own; per layer the `pre_norm` arrangement with layer norms that
have a gain and no bias.  A layer's mixer is one of three: an attention inside chunks of positions, with
short convolutions on q, k and v, a learned bias for every bucket of distances and an output gate a head; a
windowed attention with biases, a norm a head on q and k, no positions in its scores and a sink of score
zero; or a windowed attention over cached low-rank rows, rotated in neighbouring pairs, with an output gate
a value.  Where the configuration says so, a layer of the first two kinds blends its values with those that
the first such layer made for the same token.  The feed-forward is a set of ungated experts with the square
of relu, chosen by a softmax router within the best groups and weighed by the scores as they are, with a
shared expert of the same form, or absent; after it a per-layer input taken from the token ids
(`token_side_input`).  A last norm and an untied head.

The design's fixed numbers: the sink's score of zero stands here; everything else comes from the
configuration or from a tensor's shape.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.podenex import PodenexConfig
from ..parts.spec import Application, LayerSpec, ModelSpec, PartSpec

SINK_SCORE = 0.0


def _mixer(cfg: PodenexConfig, kind: str, m: dict, p: str, value_mix) -> PartSpec:
    d, eps = cfg.width, cfg.norm_eps
    if kind == "latent_attention":
        return PartSpec("latent_attention", p, {
            "width": d, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "q_rank": m["q_rank"],
            "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": eps, "window": m["mask"]["size"], "gate": "g",
            "rotary": {"dims": m["rot"]["dims"], "base": m["rot"]["base"], "interleaved": True}})
    shape = {"width": d, "n_heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
             "scale": m["scale"], "qkv": ("q", "k", "v"), "out": "o", "stored": "out_in", "bias": False, "suffix": "",
             "value_mix": value_mix}
    if kind == "attention":
        return PartSpec("causal_attention", p, {
            **shape, "conv": (m["conv"], ".conv"), "chunk": m["mask"]["size"],
            "distance_bias": ("rel", m["bias_max"], m.get("bias_rows", 32)), "gate": "g", "gate_scope": "head"})
    return PartSpec("causal_attention", p, {
        **shape, "qkv_bias": ".b", "out_bias": ".b", "qk_norm": ("q.norm", "k.norm"), "qk_norm_scope": "head", "norm_eps": eps,
        "window": m["mask"]["size"], "fixed_sink": SINK_SCORE})


def build_spec(cfg: PodenexConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("layernorm", name, {"width": d, "eps": eps, "weight": "", "bias": None})  # noqa: E731
    layers, ignored, first = [], [], None
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        value_mix = None
        if m.get("v_mix"):
            value_mix = "keep" if first is None else "vmix"      # the first one's values are kept for the others of the step
            first = i if first is None else first
        if value_mix != "vmix":
            ignored.append(rf"l{i}\.mix\.vmix")
        mlp = layer.get("mlp")
        ffn = None
        if mlp is not None:
            router, shared = mlp["router"], mlp.get("shared")
            groups = router.get("groups") or {"count": 1, "keep": 1}
            ffn = PartSpec("routed_experts", p + "mlp.", {
                "width": d, "experts": router["experts"], "top": router["top"], "inner": mlp["expert"]["ff"],
                "groups": groups["count"], "keep_groups": groups["keep"], "group_top": 1, "scores": "softmax_all",
                "correction": None, "gate": None, "activation": "relu2", "shared_inner": shared["ff"] if shared else 0})
        else:
            ignored.append(rf"l{i}\.norm2")
        addons = ()
        if cfg.side_dim:
            addons = (PartSpec("token_side_input", p, {"width": d, "vocab": cfg.vocab, "dim": cfg.side_dim, "layer": i,
                                                       "layers": len(cfg.layers), "eps": eps}),)
        layers.append(LayerSpec("pre_norm", norm(p + "norm1"), _mixer(cfg, layer["type"], m, p + "mix.", value_mix),
                                norm(p + "norm2") if ffn is not None else None, ffn, addons=addons))
    return ModelSpec(width=d, vocab_size=cfg.vocab, token_table="embed", position=PartSpec("none", ""),
                     layers=tuple(layers), schedule=tuple(Application(i) for i in range(len(layers))),
                     final_norm=norm("final.norm"), head="head", ignored_tensors=tuple(ignored))


register_architecture(PodenexConfig.architecture, PodenexConfig, build_spec)
