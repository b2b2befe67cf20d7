"""Typed configuration of the Botuvik decoder, read from config.json's own keys.

    architecture    "Botuvik"
    vocab, width
    norm.eps
    layers[]        type: which mixer the layer has; mixer: its sizes; mlp: its feed-forward, or null for none
      "attention"   mixer {heads, kv_heads (absent: heads), dim, vdim (absent: dim), scale, softcap (absent: none),
                           rot {base, dims} (absent: nothing turns)}
      "mlstm"       mixer {heads, dim, vdim, gate_cap}
      mlp {kind "dense", ff}
      mlp {kind "moe", expert {ff}, router {experts, top, groups {count, keep} (absent: none)},
           shared {ff} (absent: no shared expert)}
    loop            {start, stop, times}: layers start..stop-1 run `times` times in a row (absent: each layer once)

Every size and constant is a parameter.  The design has no table of positions and no limit of its own on a request's
length.  `initializer_range` (absent: 0.02) only serves the random-weights mode."""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Optional

from .model_config import ConfigError
from .nafevik_config import _number, _positive_int, _section

MIXER_TYPES = ("attention", "mlstm")
MLP_KINDS = ("dense", "moe")


def _attention(mixer: dict, where: str) -> None:
    heads = _positive_int(mixer.get("heads"), f"{where}.heads")
    if heads % _positive_int(mixer.get("kv_heads", heads), f"{where}.kv_heads"):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    dim = _positive_int(mixer.get("dim"), f"{where}.dim")
    _positive_int(mixer.get("vdim", dim), f"{where}.vdim")
    _number(mixer.get("scale"), f"{where}.scale", positive=False)
    if mixer.get("softcap") is not None:
        _number(mixer["softcap"], f"{where}.softcap")
    if mixer.get("rot") is not None:
        rot = _section(mixer, "rot", where)
        dims = _positive_int(rot.get("dims"), f"{where}.rot.dims")
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
        _number(rot.get("base"), f"{where}.rot.base")


def _mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind is not known; known: {MLP_KINDS}")
    if mlp["kind"] == "dense":
        _positive_int(mlp.get("ff"), f"{where}.ff")
        return
    _positive_int(_section(mlp, "expert", where).get("ff"), f"{where}.expert.ff")
    router = _section(mlp, "router", where)
    experts = _positive_int(router.get("experts"), f"{where}.router.experts")
    top = _positive_int(router.get("top"), f"{where}.router.top")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router.top exceeds the number of experts")
    if router.get("groups") is not None:
        groups = _section(router, "groups", f"{where}.router")
        count = _positive_int(groups.get("count"), f"{where}.router.groups.count")
        keep = _positive_int(groups.get("keep"), f"{where}.router.groups.keep")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"config.json: {where}.router.groups: count must divide the experts, keep be at most count, and "
                              "the kept groups hold at least `top` experts")
    if mlp.get("shared") is not None:
        _positive_int(_section(mlp, "shared", where).get("ff"), f"{where}.shared.ff")


@dataclass(frozen=True)
class BotuvikConfig:
    width: int
    vocab: int
    norm_eps: float
    layers: tuple                      # of dicts as in config.json (validated)
    loop: Optional[tuple] = None       # (start, stop, times)
    initializer_range: float = 0.02
    extra: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, raw: dict) -> "BotuvikConfig":
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
            if kind == "attention":
                _attention(mixer, where)
            else:
                for key in ("heads", "dim", "vdim"):
                    _positive_int(mixer.get(key), f"{where}.{key}")
                _number(mixer.get("gate_cap"), f"{where}.gate_cap")
            _mlp(layer.get("mlp"), f"layers[{i}].mlp")
            checked.append(copy.deepcopy(layer))
        loop = raw.get("loop")
        if loop is not None:
            if not isinstance(loop, dict):
                raise ConfigError("config.json: loop must be an object")
            start, stop, times = loop.get("start"), loop.get("stop"), loop.get("times")
            for name, value in (("start", start), ("stop", stop)):
                if isinstance(value, bool) or not isinstance(value, int) or value < 0:
                    raise ConfigError(f"config.json: loop.{name} must be a non-negative integer")
            _positive_int(times, "loop.times")
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: loop {start}..{stop} does not lie within the {len(layers)} layers")
            loop = (start, stop, times)
        known = {"architecture", "vocab", "width", "norm", "layers", "loop", "initializer_range"}
        return cls(width=width, vocab=_positive_int(raw.get("vocab"), "vocab"),
                   norm_eps=_number(_section(raw, "norm", "the model").get("eps"), "norm.eps"), layers=tuple(checked), loop=loop,
                   initializer_range=float(raw.get("initializer_range", 0.02)),
                   extra={k: v for k, v in raw.items() if k not in known})

    def to_dict(self) -> dict:
        out = {"architecture": "Botuvik", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.initializer_range != 0.02:
            out["initializer_range"] = self.initializer_range
        out.update(self.extra)
        return out

    def layer_runs(self) -> list:
        """The order in which layers run: (layer, pass of the loop or None, first of its pass)."""
        runs, n = [], len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (n, n, 0)
        runs += [(i, None, False) for i in range(start)]
        for t in range(times):
            runs += [(i, t, i == start) for i in range(start, stop)]
        return runs + [(i, None, False) for i in range(stop, n)]
