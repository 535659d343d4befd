"""Podenex's configuration, read from its own config.json.

The file is nested: `vocab`, `width`, `norm.eps`, optionally `token_side.dim` (the per-layer input taken
from the token ids), and `layers`, a list with one entry per layer: `type` (which mixer the layer has:
`attention`, `attention_2` or `latent_attention`), `mixer` (that mixer's sizes and constants) and `mlp` (the
experts', or null for a layer without a feed-forward).  The architecture is named by a top-level
`architecture` string.  Every size and constant is taken from there (the number of distance buckets is the
stored table's; `bias_rows` names it for random-weights mode); what the design knows is checked here, key by
key, so that an error names the key.
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig

MIXERS = ("attention", "attention_2", "latent_attention")
MLPS = ("moe",)


def _get(d: dict, path: str, kind, where: str):
    cur: Any = d
    for key in path.split("."):
        if not isinstance(cur, dict) or key not in cur or cur[key] is None:
            raise ConfigError(f"PodenexConfig: {where}{path} is missing")
        cur = cur[key]
    if isinstance(cur, bool) or not isinstance(cur, (int, float)) or (kind is int and int(cur) != cur):
        raise ConfigError(f"PodenexConfig: {where}{path} = {cur!r}, expected {'a whole number' if kind is int else 'a number'}")
    cur = kind(cur)
    if not cur > 0:
        raise ConfigError(f"PodenexConfig: {where}{path} = {cur} must be positive")
    return cur


@dataclasses.dataclass(frozen=True)
class PodenexConfig(ModelConfig):
    architecture: ClassVar[str] = "Podenex"

    vocab: int
    width: int
    norm_eps: float
    side_dim: int          # 0: no per-layer input from the token ids
    layers: tuple          # the entries of config.json's `layers`, checked, as plain dicts

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "PodenexConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("PodenexConfig: layers is missing or empty")
        cfg = cls(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""), norm_eps=_get(d, "norm.eps", float, ""),
                  side_dim=0 if d.get("token_side") is None else _get(d, "token_side.dim", int, ""),
                  layers=tuple(copy.deepcopy(layers)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        mixed = None           # values a token of the layers that blend theirs with the first such layer's
        for i, layer in enumerate(self.layers):
            at = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"PodenexConfig: layers[{i}] is not an object")
            if layer.get("type") not in MIXERS:
                raise ConfigError(f"PodenexConfig: {at}type = {layer.get('type')!r} is not one of {MIXERS}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"PodenexConfig: {at}mixer is missing")
            for key in ("dim", "heads", "vdim", "mask.size"):
                _get(m, key, int, at + "mixer.")
            _get(m, "scale", float, at + "mixer.")
            if layer["type"] == "latent_attention":
                for key in ("kv_rank", "q_rank", "rot_dim", "rot.dims"):
                    _get(m, key, int, at + "mixer.")
                _get(m, "rot.base", float, at + "mixer.")
                if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["rot_dim"]:
                    raise ConfigError(f"PodenexConfig: {at}mixer.rot.dims = {m['rot']['dims']} must be even and at most rot_dim")
                if m.get("v_mix"):
                    raise ConfigError(f"PodenexConfig: {at}mixer.v_mix: a latent layer's values are not blended")
            else:
                if m["heads"] % _get(m, "kv_heads", int, at + "mixer."):
                    raise ConfigError(f"PodenexConfig: {at}mixer.heads is not a multiple of kv_heads")
                if m.get("v_mix") not in (None, True, False):
                    raise ConfigError(f"PodenexConfig: {at}mixer.v_mix = {m['v_mix']!r}, expected true or false")
                if m.get("v_mix"):
                    values = m["kv_heads"] * m["vdim"]
                    if mixed not in (None, values):
                        raise ConfigError(f"PodenexConfig: {at}mixer.v_mix: {values} values a token where the first such layer "
                                          f"has {mixed}")
                    mixed = values
            if layer["type"] == "attention":
                _get(m, "conv", int, at + "mixer.")
                _get(m, "bias_max", float, at + "mixer.")
                if m.get("bias_rows") is not None and _get(m, "bias_rows", int, at + "mixer.") < 2:
                    raise ConfigError(f"PodenexConfig: {at}mixer.bias_rows = {m['bias_rows']} must be at least 2")
            self._check_mlp(layer.get("mlp"), at)

    @staticmethod
    def _check_mlp(mlp, at: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in MLPS:
            raise ConfigError(f"PodenexConfig: {at}mlp.kind = {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} "
                              f"is not one of {MLPS}")
        _get(mlp, "expert.ff", int, at + "mlp.")
        experts = _get(mlp, "router.experts", int, at + "mlp.")
        top = _get(mlp, "router.top", int, at + "mlp.")
        if top > experts:
            raise ConfigError(f"PodenexConfig: {at}mlp.router.top = {top} is more than its {experts} experts")
        if mlp["router"].get("groups") is not None:
            count = _get(mlp, "router.groups.count", int, at + "mlp.")
            keep = _get(mlp, "router.groups.keep", int, at + "mlp.")
            if experts % count or keep > count or keep * (experts // count) < top:
                raise ConfigError(f"PodenexConfig: {at}mlp.router.groups = {count} groups, {keep} kept, do not fit "
                                  f"{experts} experts of which {top} are chosen")
        if mlp.get("shared") is not None:
            _get(mlp, "shared.ff", int, at + "mlp.")

    def check_dtype(self, dtype: str) -> None:
        """Nothing is refused: every part of this design has a kernel for every size in both compute types (rows
        that are no multiples of 16 bytes take the slower ones)."""

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": copy.deepcopy(list(self.layers))}
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        return d
