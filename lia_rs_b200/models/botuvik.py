"""Botuvik: a decoder whose layers carry an RMS norm before and after each sublayer and whose mixer is, layer by layer,
grouped-query softmax attention (biases on q, k and v, interleaved rotary pairs, a weightless norm of every head behind
them, a tanh cap on the scores, a learned sink per head) or the matrix memory of xLSTM.  The feed-forward is a dense
squared ReLU, a mixture of gated SiLU experts (sigmoid scores, groups judged by their two largest, weights renormalised
over the chosen, a shared expert that every token uses), or absent.  A run of layers may be gone through several times
with the same weights, each pass with caches and states of its own: a stored vector is added to the stream ahead of every
pass, the embedding output ahead of every pass but the first.  A final RMS norm and an untied head.  This file only
translates a `BotuvikConfig` into a `ModelSpec`: every mechanism is a registered part.

Checkpoint names: embed, loop.step, l<i>.norm1, l<i>.norm1b, l<i>.norm2, l<i>.norm2b, l<i>.mix.*, l<i>.mlp.*, final.norm,
head."""
from __future__ import annotations

from ..config import BotuvikConfig, register_architecture
from ..parts import LayerSpec, PartSpec
from .decoder import ModelSpec, ScheduleEntry


def build_botuvik(config: BotuvikConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = PartSpec("rmsnorm", {"hidden": width, "eps": eps, "tensor": ""})
    layers = []
    for layer in config.layers:
        m = layer["mixer"]
        if layer["type"] == "attention":
            mixer = PartSpec("sink_attention", {
                "hidden": width, "heads": m["heads"], "kv_heads": m.get("kv_heads", m["heads"]), "head_dim": m["dim"],
                "v_head_dim": m.get("vdim", m["dim"]), "scale": m["scale"], "softcap": m.get("softcap"), "rot": m.get("rot"),
                "rot_pairs": True, "biases": "qkv", "qk_norm": "behind", "norm_eps": eps, "sink": "learned"})
        else:
            mixer = PartSpec("mlstm", {"hidden": width, "heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
                                       "gate_cap": m["gate_cap"], "norm_eps": eps})
        mlp = layer.get("mlp")
        if mlp is None:
            feed_forward = None
        elif mlp["kind"] == "dense":
            feed_forward = PartSpec("dense_act", {"hidden": width, "intermediate": mlp["ff"], "activation": "relu_squared",
                                                  "names": {"up": "up", "down": "down"}})
        else:
            router, shared = mlp["router"], mlp.get("shared")
            feed_forward = PartSpec("expert_mixture", {
                "hidden": width, "experts": router["experts"], "top": router["top"], "router_scale": 1.0,
                "intermediate": mlp["expert"]["ff"], "scores": "sigmoid", "groups": router.get("groups"),
                "group_score": "two_best", "renormalise": True, "shared": {"intermediate": shared["ff"]} if shared else None,
                "shared_gated": False})
        layers.append(LayerSpec(
            mixer=mixer, feed_forward=feed_forward, norm=norm, arrangement="sandwich",
            names={"norm1": "norm1", "norm1b": "norm1b", "norm2": "norm2", "norm2b": "norm2b", "mixer": "mix.",
                   "feed_forward": "mlp."}))
    schedule, junctions = [], {}
    for position, (layer, loop_pass, first_of_pass) in enumerate(config.layer_runs()):
        # every run of a layer has a cache (attention) or a state (the memory) of its own
        schedule.append(ScheduleEntry(layer, cache=position if config.layers[layer]["type"] == "attention" else None))
        if first_of_pass:
            junctions[position] = PartSpec("stream_step", {"hidden": width, "row": loop_pass, "rows": config.loop[2],
                                                           "first": loop_pass > 0, "names": {"bias": "loop.step"}})
    return ModelSpec(hidden_size=width, vocab_size=config.vocab, max_positions=None, layers=layers, final_norm=norm,
                     schedule=schedule, junctions=junctions, embedding_name="embed", head_name="head", layer_prefix="l{}.",
                     final_norm_prefix="final.norm")


register_architecture(("Botuvik",), BotuvikConfig, build_botuvik)
