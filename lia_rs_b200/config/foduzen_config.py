"""Typed configuration of the Foduzen decoder, read from config.json's own keys.

    architecture    "Foduzen"
    vocab, width
    norm.eps
    embedding.scale the embedding output's factor (absent: 1)
    layers[]        type: which mixer the layer has; mixer: its sizes; mlp {kind "dense", ff} or null for none
      "rglru"       mixer {width, blocks, conv}
      "parallel"    mixer {left {heads, kv_heads (absent: heads), dim, vdim (absent: dim), scale, mask {size} (absent: every
                                 earlier key is seen)},
                           right {heads, vdim, state, groups (absent: 1), norm_groups (absent: 1), conv}}

Every size and constant is a parameter.  Positions enter through a sinusoidal vector added to the embedding, so the design
has no table of positions and no limit of its own on a request's length.  `initializer_range` (absent: 0.02) only serves the
random-weights mode."""
from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .model_config import ConfigError
from .nafevik_config import _number, _positive_int, _section

MIXER_TYPES = ("rglru", "parallel")
MLP_KINDS = ("dense",)


def _left(left: dict, where: str) -> None:
    heads = _positive_int(left.get("heads"), f"{where}.heads")
    if heads % _positive_int(left.get("kv_heads", heads), f"{where}.kv_heads"):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    _positive_int(left.get("vdim", _positive_int(left.get("dim"), f"{where}.dim")), f"{where}.vdim")
    _number(left.get("scale"), f"{where}.scale", positive=False)
    if left.get("mask") is not None:
        _positive_int(_section(left, "mask", where).get("size"), f"{where}.mask.size")


def _right(right: dict, where: str) -> None:
    for key in ("heads", "vdim", "state", "conv"):
        _positive_int(right.get(key), f"{where}.{key}")
    if right["heads"] % _positive_int(right.get("groups", 1), f"{where}.groups"):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of groups")
    if (right["heads"] * right["vdim"]) % _positive_int(right.get("norm_groups", 1), f"{where}.norm_groups"):
        raise ConfigError(f"config.json: {where}.heads * vdim must be a multiple of norm_groups")


@dataclass(frozen=True)
class FoduzenConfig:
    width: int
    vocab: int
    norm_eps: float
    layers: tuple                      # of dicts as in config.json (validated)
    embedding_scale: float = 1.0
    initializer_range: float = 0.02
    extra: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, raw: dict) -> "FoduzenConfig":
        width = _positive_int(raw.get("width"), "width")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            if not isinstance(layer, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not known; known: {MIXER_TYPES}")
            where = f"layers[{i}].mixer"
            mixer = _section(layer, "mixer", f"layers[{i}]")
            if kind == "rglru":
                for key in ("width", "blocks", "conv"):
                    _positive_int(mixer.get(key), f"{where}.{key}")
                if mixer["width"] % mixer["blocks"]:
                    raise ConfigError(f"config.json: {where}.width must be a multiple of blocks")
            else:
                _left(_section(mixer, "left", where), f"{where}.left")
                _right(_section(mixer, "right", where), f"{where}.right")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
                    raise ConfigError(f"config.json: layers[{i}].mlp.kind is not known; known: {MLP_KINDS}")
                _positive_int(mlp.get("ff"), f"layers[{i}].mlp.ff")
            checked.append(copy.deepcopy(layer))
        embedding = raw.get("embedding") or {}
        known = {"architecture", "vocab", "width", "norm", "layers", "embedding", "initializer_range"}
        return cls(width=width, vocab=_positive_int(raw.get("vocab"), "vocab"),
                   norm_eps=_number(_section(raw, "norm", "the model").get("eps"), "norm.eps"), layers=tuple(checked),
                   embedding_scale=_number(embedding.get("scale", 1.0), "embedding.scale", positive=False),
                   initializer_range=float(raw.get("initializer_range", 0.02)),
                   extra={k: v for k, v in raw.items() if k not in known})

    def to_dict(self) -> dict:
        out = {"architecture": "Foduzen", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers))}
        if self.initializer_range != 0.02:
            out["initializer_range"] = self.initializer_range
        out.update(self.extra)
        return out
