"""Mamusun's configuration, read from its own config.json.

The file is nested: `vocab`, `width`, `norm.eps`, `postln_alpha` (the factor on the stream in every sum that a norm
follows), and `layers`, a list with one entry per layer: `type` (which mixer the layer has: `attention`, `attention_2`
or `parallel`), `mixer` (that mixer's sizes and constants) and `mlp` (the feed-forward's: `kind` dense or moe, or null
for a layer without one).  An `attention` layer with `kv_from` reads the keys and values of an earlier one.  The
architecture is named by a top-level `architecture` string.  Every size and constant is taken from there and checked
here, key by key, so that an error names the key.
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig

MIXERS = ("attention", "attention_2", "parallel")
MLPS = ("dense", "moe")


def _get(d: dict, path: str, kind, where: str, positive: bool = True):
    cur: Any = d
    for key in path.split("."):
        if not isinstance(cur, dict) or key not in cur or cur[key] is None:
            raise ConfigError(f"MamusunConfig: {where}{path} is missing")
        cur = cur[key]
    if isinstance(cur, bool) or not isinstance(cur, (int, float)) or (kind is int and int(cur) != cur):
        raise ConfigError(f"MamusunConfig: {where}{path} = {cur!r}, expected {'a whole number' if kind is int else 'a number'}")
    cur = kind(cur)
    if positive and not cur > 0:
        raise ConfigError(f"MamusunConfig: {where}{path} = {cur} must be positive")
    return cur


@dataclasses.dataclass(frozen=True)
class MamusunConfig(ModelConfig):
    architecture: ClassVar[str] = "Mamusun"

    vocab: int
    width: int
    norm_eps: float
    alpha: float
    layers: tuple          # the entries of config.json's `layers`, checked, as plain dicts

    def __hash__(self):
        return hash((self.vocab, self.width, self.norm_eps, self.alpha, len(self.layers)))

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "MamusunConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("MamusunConfig: layers is missing or empty")
        cfg = cls(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""), norm_eps=_get(d, "norm.eps", float, ""),
                  alpha=_get(d, "postln_alpha", float, "", positive=False), layers=tuple(copy.deepcopy(layers)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            at = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"MamusunConfig: layers[{i}] is not an object")
            if layer.get("type") not in MIXERS:
                raise ConfigError(f"MamusunConfig: {at}type = {layer.get('type')!r} is not one of {MIXERS}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"MamusunConfig: {at}mixer is missing")
            if layer["type"] == "parallel":
                if not isinstance(m.get("left"), dict):
                    raise ConfigError(f"MamusunConfig: {at}mixer.left is missing")
                self._check_heads(m["left"], at + "mixer.left.")
                _get(m["left"], "mask.size", int, at + "mixer.left.")
                self._check_rotation(m["left"], at + "mixer.left.", ("factor", "low", "high", "original"))
                for key in ("blocks", "conv", "width"):
                    _get(m, "right." + key, int, at + "mixer.")
                if m["right"]["width"] % m["right"]["blocks"]:
                    raise ConfigError(f"MamusunConfig: {at}mixer.right.width is not a multiple of blocks")
            else:
                self._check_heads(m, at + "mixer.")
                if layer["type"] == "attention":
                    _get(m, "mask.size", int, at + "mixer.")
                    self._check_source(i, m, at + "mixer.")
                else:
                    self._check_rotation(m, at + "mixer.", ("factor", "fast", "slow", "original"))
                    if m["vdim"] != m["dim"]:
                        raise ConfigError(f"MamusunConfig: {at}mixer.vdim = {m['vdim']}: values that are keys have their dim {m['dim']}")
            self._check_mlp(layer.get("mlp"), at + "mlp.")

    @staticmethod
    def _check_heads(m: dict, at: str) -> None:
        for key in ("dim", "heads", "kv_heads", "vdim"):
            _get(m, key, int, at)
        _get(m, "scale", float, at)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"MamusunConfig: {at}heads is not a multiple of kv_heads")

    @staticmethod
    def _check_rotation(m: dict, at: str, scaling) -> None:
        _get(m, "rot.dims", int, at)
        _get(m, "rot.base", float, at)
        if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]:
            raise ConfigError(f"MamusunConfig: {at}rot.dims = {m['rot']['dims']} must be even and at most dim")
        if m["rot"].get("scaling") is not None:
            for key in scaling:
                _get(m, "rot.scaling." + key, float, at)

    def _check_source(self, i: int, m: dict, at: str) -> None:
        src = m.get("kv_from")
        if src is None:
            return
        if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
            raise ConfigError(f"MamusunConfig: {at}kv_from = {src!r} must name an earlier layer")
        other = self.layers[src]
        if other.get("type") != "attention" or other["mixer"].get("kv_from") is not None:
            raise ConfigError(f"MamusunConfig: {at}kv_from = {src} names a layer without keys and values of its own")
        for key in ("kv_heads", "dim", "vdim"):
            if other["mixer"].get(key) != m.get(key):
                raise ConfigError(f"MamusunConfig: {at}kv_from = {src}: the two layers differ in {key}")

    @staticmethod
    def _check_mlp(mlp, at: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in MLPS:
            raise ConfigError(f"MamusunConfig: {at}kind = {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not one of {MLPS}")
        if mlp["kind"] == "dense":
            _get(mlp, "ff", int, at)
            return
        _get(mlp, "expert.ff", int, at)
        _get(mlp, "expert.limit", float, at)
        if _get(mlp, "router.top", int, at) > _get(mlp, "router.experts", int, at):
            raise ConfigError(f"MamusunConfig: {at}router.top = {mlp['router']['top']} is more than its {mlp['router']['experts']} experts")

    def check_dtype(self, dtype: str) -> None:
        """Nothing is refused: every part of this design has a kernel for every size in both compute types (rows
        that are no multiples of 16 bytes take the slower ones)."""

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "postln_alpha": self.alpha, "layers": copy.deepcopy(list(self.layers))}
