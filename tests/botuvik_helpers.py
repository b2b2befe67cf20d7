"""Tiny Botuvik configurations for the tests, their model folders with random weights, and the comparison with the plain
implementation (tests/plain_botuvik.py).

The configurations differ in everything that config.json gives: widths and vocabularies; the order of the two kinds of layer
(each first, last and alone); a run of layers gone through once, twice and three times, at the start, in the middle, at the
end, over one layer, several and all, and no such run; attention with as many key heads as query heads, fewer, and one, key
and value sizes equal and unequal, partial, full and absent rotation, a cap present and absent; memories with 1 to 5 heads,
key and value sizes that are not multiples of four, small and large caps of the gates; dense feed-forwards, mixtures of 1 to
12 experts of which 1 to all are chosen, groups of one, two and more experts present and absent with 1 to all kept, with and
without a shared expert; layers without a feed-forward."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_botuvik


def _attention(heads, kv_heads, dim, vdim, scale, softcap=None, rot=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        mixer["softcap"] = softcap
    if rot:
        mixer["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _mlstm(heads, dim, vdim, gate_cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


BOTUVIK = {
    "bot-A": dict(          # a run in the middle, odd sizes that no 16-byte access fits
        config={"architecture": "Botuvik", "vocab": 97, "width": 60, "norm": {"eps": 2e-5}, "initializer_range": 0.08,
                "layers": [
                    _mlstm(3, 10, 14, 9.0, _moe(36, 6, 2, groups=(3, 2), shared=20)),
                    _attention(4, 2, 20, 12, 0.25, softcap=6.0, rot=(1000.0, 12), mlp=_dense(50)),
                    _mlstm(1, 24, 6, 15.0, None),
                    _attention(3, 3, 16, 16, 0.4, softcap=20.0, rot=(5e4, 16), mlp=_moe(24, 5, 5, shared=None))],
                "loop": {"start": 1, "stop": 3, "times": 3}},
        seed=11, page_size=8),
    "bot-B": dict(          # attention first, no run, no cap, no rotation, one expert a group
        config={"architecture": "Botuvik", "vocab": 131, "width": 96, "norm": {"eps": 3e-6}, "initializer_range": 0.06,
                "layers": [
                    _attention(6, 1, 24, 40, 0.3, mlp=_moe(40, 4, 1, groups=(4, 2), shared=64)),
                    _attention(2, 2, 8, 8, 0.5, softcap=3.0, rot=(100.0, 4), mlp=None),
                    _mlstm(5, 16, 16, 4.0, _dense(72))]},
        seed=12, page_size=4),
    "bot-C": dict(          # sizes of real shapes' divisibility: the tensor-core kernels serve every mechanism; all layers run twice
        config={"architecture": "Botuvik", "vocab": 211, "width": 128, "norm": {"eps": 1e-6}, "initializer_range": 0.05,
                "layers": [
                    _mlstm(2, 64, 128, 12.0, _moe(64, 12, 3, groups=(4, 2), shared=128)),
                    _attention(4, 1, 64, 64, 0.2, softcap=25.0, rot=(1e5, 64), mlp=_dense(192)),
                    _attention(4, 2, 64, 128, 0.15, softcap=12.0, rot=(1e4, 32), mlp=_moe(96, 8, 2, groups=(2, 1)))],
                "loop": {"start": 0, "stop": 3, "times": 2}},
        seed=13, page_size=16),
    "bot-D": dict(          # memories alone: no pages anywhere; a run of one pass at the end
        config={"architecture": "Botuvik", "vocab": 157, "width": 80, "norm": {"eps": 1e-5}, "initializer_range": 0.07,
                "layers": [_mlstm(2, 32, 48, 6.0, _dense(100)), _mlstm(4, 16, 32, 20.0, _moe(48, 1, 1, shared=32)),
                           _mlstm(1, 48, 160, 10.0, None)],
                "loop": {"start": 2, "stop": 3, "times": 1}},
        seed=14, page_size=16),
    "bot-F": dict(          # tensor-core sizes without a router (no row rests on a close call); the run is the first two layers
        config={"architecture": "Botuvik", "vocab": 160, "width": 96, "norm": {"eps": 1e-5}, "initializer_range": 0.06,
                "layers": [
                    _mlstm(3, 32, 64, 18.0, _dense(128)),
                    _attention(8, 2, 128, 128, 0.1, softcap=30.0, rot=(2e4, 64), mlp=None),
                    _mlstm(1, 16, 256, 7.0, _dense(64))],
                "loop": {"start": 0, "stop": 2, "times": 2}},
        seed=16, page_size=16),
    "bot-E": dict(          # attention alone; the run is the last layer, gone through twice
        config={"architecture": "Botuvik", "vocab": 113, "width": 72, "norm": {"eps": 1e-5}, "initializer_range": 0.07,
                "layers": [_attention(8, 2, 32, 32, 0.25, softcap=8.0, rot=(2e3, 32), mlp=_dense(90)),
                           _attention(3, 1, 128, 128, 0.12, softcap=15.0, rot=(1e6, 64), mlp=_moe(32, 9, 4, groups=(3, 2), shared=40))],
                "loop": {"start": 1, "stop": 2, "times": 2}},
        seed=15, page_size=16),
}


def random_configuration(seed: int) -> dict:
    """A configuration drawn at random: 2 to 4 layers of both kinds in any order, sizes that are and are not multiples of 4,
    8 or 16, every optional key present or absent."""
    import random
    rng = random.Random(seed)
    width = rng.choice([48, 64, 72, 96, 128, 144])
    if seed % 3 == 0:
        width = rng.choice([50, 66, 100, 257])          # rows that no 16-byte access fits
    layers = []
    for _ in range(rng.randint(2, 4)):
        kind = rng.choice(["none", "dense", "moe", "moe"])
        mlp = None
        if kind == "dense":
            mlp = _dense(rng.choice([40, 96, 100, 200]))
        elif kind == "moe":
            count = rng.choice([None, 1, 2, 3])
            experts = (count or 1) * rng.choice([1, 2, 3, 4])
            keep = rng.randint(1, count) if count else None
            top = rng.randint(1, min(4, (keep * (experts // count)) if count else experts))
            mlp = _moe(rng.choice([16, 30, 48, 64]), experts, top, groups=(count, keep) if count else None,
                       shared=rng.choice([None, 24, 80]))
        if rng.random() < 0.5:
            layers.append(_mlstm(rng.choice([1, 2, 3, 4]), rng.choice([6, 8, 16, 18, 32, 64, 80]), rng.choice([8, 12, 16, 30, 64, 144]),
                                 rng.choice([3.0, 8.0, 15.0, 30.0]), mlp))
            continue
        kv_heads = rng.choice([1, 2, 3])
        dim = rng.choice([8, 16, 24, 32, 40, 64])
        rot = rng.choice([None, (rng.choice([100.0, 1e4, 1e6]), rng.choice([2, dim // 2 // 2 * 2, dim]))])
        layer = _attention(kv_heads * rng.choice([1, 2, 4]), kv_heads, dim, rng.choice([8, 16, 24, 32, 64, dim]), rng.uniform(0.1, 0.5),
                           softcap=rng.choice([None, 2.0, 10.0, 40.0]), rot=rot, mlp=mlp)
        if rng.random() < 0.4:
            m = layer["mixer"]
            if m["kv_heads"] == m["heads"]:
                m.pop("kv_heads")
            if m["vdim"] == m["dim"]:
                m.pop("vdim")
        layers.append(layer)
    config = {"architecture": "Botuvik", "vocab": rng.choice([61, 128, 250]), "width": width,
              "norm": {"eps": rng.choice([1e-6, 1e-5, 3e-5])}, "initializer_range": 0.07, "layers": layers}
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        config["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.choice([1, 2, 2, 3])}
    return config


def make_model(folder: str, name: str) -> dict:
    """The folder through the package's random-weights mode; then the weights are moved to where a fault shows: queries and keys
    are normed by the design, so their scale is what config gives, and the biases of q, k and v are of order one; the sinks
    lie between "takes nothing" and "takes most"; every norm weight is spread; the memories' forget gates reach from "forgets
    within a few tokens" to "keeps hundreds", their input gates are of both signs; the router's rows are raised; the vectors
    ahead of a pass are of the stream's size.  Returns {dir, config, weights (by checkpoint name, as stored), page_size, name}."""
    from safetensors.torch import load_file, save_file

    from lia_rs_b200.config import BotuvikConfig
    from lia_rs_b200.weights import write_random_model
    if name in BOTUVIK:
        entry = BOTUVIK[name]
    else:
        seed = int(name.split("-")[1])
        entry = dict(config=random_configuration(seed), seed=seed, page_size=(4, 8, 16)[seed % 3])
    write_random_model(BotuvikConfig.from_dict(entry["config"]), folder, seed=entry["seed"])
    path = os.path.join(folder, "model.safetensors")
    weights = load_file(path)
    g = torch.Generator().manual_seed(entry["seed"] + 100)
    bf16 = lambda t: t.to(torch.bfloat16)
    for key in list(weights):
        shape = weights[key].shape
        tail = key.split(".", 1)[1] if "." in key else key
        normal = lambda: torch.randn(shape, generator=g)
        if "norm" in tail:
            weights[key] = bf16(1.0 + 0.3 * normal())
        elif key == "embed":
            weights[key] = bf16(0.7 * normal())
        elif key == "loop.step":
            weights[key] = bf16(0.5 * normal())
        elif tail == "mix.sink":
            weights[key] = bf16(1.0 + 2.0 * normal())
        elif tail == "mix.f.b":
            weights[key] = bf16(5.0 + 2.5 * normal())
        elif tail == "mix.i.b":
            weights[key] = bf16(-1.0 + 2.0 * normal())
        elif tail in ("mix.i", "mix.f", "mlp.router"):
            weights[key] = bf16({"mix.i": 1.5, "mix.f": 0.7, "mlp.router": 2.0}[tail] * normal() / shape[-1] ** 0.5)
        elif tail in ("mix.q", "mix.k", "mix.v", "mix.g"):
            weights[key] = bf16(normal() / shape[-1] ** 0.5)
        elif tail.endswith(".b"):
            weights[key] = bf16(0.5 * normal())
    save_file(weights, path)
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    return dict(dir=folder, config=config, weights=weights, page_size=entry["page_size"], name=name)


_CACHE = {}
_MARKS = {}       # storage of a cached reference -> per row 0 (sound), 1 (behind a fragile row of its sequence), 2 (fragile)


def plain_logits(model: dict, tokens) -> torch.Tensor:
    key = (model["name"], model["dir"], tuple(tokens))
    if key not in _CACHE:
        fragile = torch.zeros(len(tokens), dtype=torch.bool)
        logits = plain_botuvik.forward(model["config"], model["weights"], list(tokens), fragile=fragile).contiguous()
        behind = (torch.cumsum(fragile.long(), 0) - fragile.long()) > 0
        _MARKS[logits.untyped_storage().data_ptr()] = torch.where(fragile, 2, behind.long())
        _CACHE[key] = logits
    return _CACHE[key]


def marks_of(reference: torch.Tensor):
    """The marks of the rows of a cached reference or of a slice of rows of one (a view of it), else None."""
    marks = _MARKS.get(reference.untyped_storage().data_ptr())
    if marks is None or reference.dim() != 2 or reference.stride(1) != 1:
        return None
    first = reference.storage_offset() // reference.stride(0)
    return marks[first:first + reference.shape[0]]


def layer_runs(config: dict) -> list:
    return [config["layers"][i] for i, _, _ in plain_botuvik.layer_order(config)]


def longest_sum(config: dict) -> int:
    sizes = [config["width"]]
    for layer in config["layers"]:
        m, mlp = layer["mixer"], layer.get("mlp")
        sizes.append(m["heads"] * max(m["dim"], m.get("vdim", m["dim"])))
        if mlp:
            sizes.append(mlp["ff"] if mlp["kind"] == "dense" else max(mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0)))
    return max(sizes)


def assert_close(actual, reference, dtype: str, what: str, config: dict):
    """Against the exact (64-bit) model.  32-bit: every logit within 8 K 2^-24 of the largest logit per layer run that the
    sums pass through (K the model's longest sum; a memory, whose sums run along the sequence, counts as four).  bfloat16:
    every row's root-mean-square error within 2.5e-2 of the largest logit, times the root of the number of layer runs
    (rounding noise of a layer adds to that of the layers before), and no single logit further off than three times that.  A
    row that the plain implementation marks as resting on a close call (a router's choice between two experts or two groups
    of nearly equal score, a memory asked for almost nothing that it holds) may come out on the other side in 16-bit arithmetic: it only has to be finite, and the rows behind
    it in its sequence, which read what it left, get four times the limit."""
    marks = marks_of(reference) if dtype != "float32" else None
    actual = torch.as_tensor(np.asarray(actual), dtype=torch.float64)
    reference = reference.to(torch.float64)
    assert actual.shape == reference.shape, f"{what}: shape {tuple(actual.shape)} vs {tuple(reference.shape)}"
    assert torch.isfinite(actual).all(), f"{what}: non-finite logits"
    runs = layer_runs(config)
    weighted = len(runs) + 3 * sum(1 for layer in runs if layer["type"] == "mlstm")
    scale = max(1.0, float(reference.abs().max()))
    error = (actual - reference).abs()
    if dtype == "float32":
        limit = 8.0 * longest_sum(config) * 2.0 ** -24 * scale * weighted
        worst = float(error.max())
    else:
        limit = 2.5e-2 * scale * max(1.0, len(runs) ** 0.5)
        if marks is not None and error.dim() == 2:
            error = error * torch.tensor([1.0, 0.25, 0.0], dtype=torch.float64)[marks][:, None]
        worst = max(float((error ** 2).mean(dim=-1).sqrt().max()), float(error.max()) / 3.0)
    if worst > limit:
        row = int(error.max(dim=-1).values.argmax()) if error.dim() > 1 else 0
        raise AssertionError(f"{what}: error {worst:.3e} > {limit:.3e} (largest at wanted row {row})")
