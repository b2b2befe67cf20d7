"""Foduzen: a decoder whose sublayers read the residual stream itself and whose outputs are normed before they join it (RMS
norms with one stored number each), with a sinusoidal vector of the position added to the scaled embedding.  The mixer is,
layer by layer, a gated linear recurrent unit behind a short convolution, or two mixers side by side, each normed and half
their sum taken: windowed grouped-query softmax attention (biases, a norm per q and k head, no rotation, a sigmoid gate on
the heads' output) and a state-space recurrence with one decay per token and head.  The feed-forward is dense with the xIELU
activation, or absent.  A final norm and an untied head.  This file only translates a `FoduzenConfig` into a `ModelSpec`:
every mechanism is a registered part.

Checkpoint names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.* (l<i>.mix.left.*, l<i>.mix.right.*), l<i>.mlp.{up,down,act},
final.norm, head."""
from __future__ import annotations

from ..config import FoduzenConfig, register_architecture
from ..parts import LayerSpec, PartSpec
from .decoder import ModelSpec

POSITION_BASE = 10000.0          # of the sinusoidal vector: fixed by the design


def build_foduzen(config: FoduzenConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = PartSpec("rmsnorm", {"hidden": width, "eps": eps, "tensor": "", "single": True})
    layers = []
    for layer in config.layers:
        m = layer["mixer"]
        if layer["type"] == "rglru":
            mixer = PartSpec("rglru", {"hidden": width, "width": m["width"], "blocks": m["blocks"], "taps": m["conv"]})
        else:
            left, right = m["left"], m["right"]
            attention = {
                "hidden": width, "heads": left["heads"], "kv_heads": left.get("kv_heads", left["heads"]),
                "head_dim": left["dim"], "v_head_dim": left.get("vdim", left["dim"]), "scale": left["scale"],
                "window": left["mask"]["size"] if left.get("mask") else None, "biases": True, "qk_norm": True,
                "norm_eps": eps, "gate": "sigmoid"}
            recurrence = {
                "hidden": width, "heads": right["heads"], "size": right["vdim"], "state": right["state"],
                "groups": right.get("groups", 1), "norm_groups": right.get("norm_groups", 1), "taps": right["conv"],
                "norm_eps": eps}
            side = lambda name: {"tensor": f"{name}.out", "hidden": width, "eps": eps}
            mixer = PartSpec("side_by_side", {"members": [
                {"kind": "sink_attention", "params": attention, "prefix": "left.", "scale": 0.5, "norm": side("left")},
                {"kind": "state_space", "params": recurrence, "prefix": "right.", "scale": 0.5, "norm": side("right")}]})
        mlp = layer.get("mlp")
        feed_forward = None if mlp is None else PartSpec("dense_act", {
            "hidden": width, "intermediate": mlp["ff"], "activation": "xielu", "names": {"up": "up", "down": "down", "act": "act"}})
        layers.append(LayerSpec(mixer=mixer, feed_forward=feed_forward, norm=norm, arrangement="postnorm",
                                names={"norm1": "norm1", "norm2": "norm2", "mixer": "mix.", "feed_forward": "mlp."}))
    return ModelSpec(hidden_size=width, vocab_size=config.vocab, max_positions=None, layers=layers, final_norm=norm,
                     embedding_scale=config.embedding_scale, embedding_name="embed", head_name="head", layer_prefix="l{}.",
                     final_norm_prefix="final.norm", sinusoidal_base=POSITION_BASE)


register_architecture(("Foduzen",), FoduzenConfig, build_foduzen)
