"""Tiny Foduzen configurations for the tests, their model folders with random weights, and the comparison with the plain
implementation (tests/plain_foduzen.py).

The configurations differ in everything that config.json gives: widths and vocabularies; the order of the two kinds of layer
(each first, last and alone); recurrent units wider and narrower than the model with 1 to 6 parts, parts that are and are not
multiples of 8 channels, 1 to 8 taps; attention with as many key heads as query heads, fewer, and one, key and value heads of
equal and of different sizes, windows of 1 token, of a few, of more than any test's length, and none; state-space recurrences
with 1 to 8 heads in 1 to 8 groups, sizes and states that are not multiples of four, norms in 1 to 8 parts that do and do not
follow the heads; layers without a feed-forward; factors on the embedding present and absent."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_foduzen


def _rglru(width, blocks, conv, ff):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": _dense(ff)}


def _dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def _left(heads, kv_heads, dim, vdim, scale, window=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        left["mask"] = {"size": window}
    return left


def _right(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def _parallel(left, right, ff):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": _dense(ff)}


FODUZEN = {
    "fod-A": dict(
        config={"architecture": "Foduzen", "vocab": 97, "width": 64, "norm": {"eps": 1e-5}, "initializer_range": 0.08,
                "embedding": {"scale": 6.0},
                "layers": [
                    _rglru(96, 3, 4, 80),
                    _parallel(_left(4, 2, 16, 24, 0.25, window=11), _right(4, 12, 20, 2, 4, 3), 96),
                    _rglru(48, 1, 2, None),
                    _parallel(_left(3, 3, 24, 8, 0.2, window=33), _right(3, 8, 6, 1, 1, 5), 40)]},
        seed=1, page_size=8),
    "fod-B": dict(          # parallel first and alone at the end, no factor, no window in one layer, a window of one token in another
        config={"architecture": "Foduzen", "vocab": 131, "width": 96, "norm": {"eps": 3e-6}, "initializer_range": 0.06,
                "layers": [
                    _parallel(_left(6, 1, 16, 12, 0.3), _right(1, 32, 32, 1, 2, 4), 120),
                    _rglru(60, 6, 1, 64),                       # parts of 10 channels, a single tap
                    _parallel(_left(2, 2, 8, 40, 0.35, window=1), _right(8, 6, 10, 8, 3, 8), None)]},
        seed=2, page_size=4),
    "fod-C": dict(          # sizes of real shapes' divisibility: the tensor-core kernels serve every mechanism
        config={"architecture": "Foduzen", "vocab": 211, "width": 128, "norm": {"eps": 1e-6}, "initializer_range": 0.05,
                "embedding": {"scale": 11.0},
                "layers": [
                    _parallel(_left(4, 1, 64, 64, 0.125, window=48), _right(4, 64, 64, 2, 1, 4), 192),
                    _rglru(192, 2, 4, 256),
                    _parallel(_left(4, 2, 64, 128, 0.13, window=20), _right(2, 32, 128, 1, 2, 4), 128),
                    _parallel(_left(2, 2, 128, 64, 0.09, window=130), _right(4, 128, 16, 4, 4, 2), 64)]},
        seed=3, page_size=16),
    "fod-D": dict(          # recurrent units alone: no pages anywhere
        config={"architecture": "Foduzen", "vocab": 157, "width": 80, "norm": {"eps": 2e-5}, "initializer_range": 0.07,
                "embedding": {"scale": 2.0},
                "layers": [_rglru(128, 2, 4, 100), _rglru(72, 4, 3, 100), _rglru(264, 3, 8, None)]},
        seed=4, page_size=16),
    "fod-W": dict(          # windows alone: the recurrent side's share is weighted with zero
        config={"architecture": "Foduzen", "vocab": 113, "width": 72, "norm": {"eps": 1e-5}, "initializer_range": 0.07,
                "embedding": {"scale": 4.0},
                "layers": [
                    _parallel(_left(4, 2, 32, 64, 0.25, window=19), _right(2, 8, 8, 1, 1, 2), 90),
                    _parallel(_left(2, 2, 64, 64, 0.2, window=64), _right(2, 8, 8, 2, 2, 2), 60),
                    _parallel(_left(3, 1, 24, 16, 0.3, window=5), _right(2, 8, 8, 1, 4, 2), None)]},
        seed=5, page_size=16, mute_right=True),
}


def random_configuration(seed: int) -> dict:
    """A configuration drawn at random: 2 to 5 layers of both kinds in any order, sizes that are and are not multiples of 4,
    8 or 16, every optional key present or absent."""
    import random
    rng = random.Random(seed)
    width = rng.choice([48, 64, 72, 96, 128, 144])
    if seed % 3 == 0:
        width = rng.choice([50, 66, 100, 257])          # rows that no 16-byte access fits
    layers = []
    for _ in range(rng.randint(2, 5)):
        ff = rng.choice([None, 40, 96, 100, 200])
        if rng.random() < 0.5:
            blocks = rng.choice([1, 2, 3, 5])
            layers.append(_rglru(blocks * rng.choice([8, 16, 18, 40, 64, 72]), blocks, rng.choice([1, 2, 3, 4, 4, 7]), ff))
            continue
        kv_heads = rng.choice([1, 2, 3])
        dim = rng.choice([8, 16, 24, 32, 40, 64])
        left = _left(kv_heads * rng.choice([1, 2, 4]), kv_heads, dim, rng.choice([8, 16, 24, 32, 64, 128, dim]), rng.uniform(0.1, 0.4),
                     window=rng.choice([None, 1, 3, 8, 17, 32, 50, 200]))
        groups = rng.choice([1, 2, 3])
        heads, vdim = groups * rng.choice([1, 2, 4]), rng.choice([6, 8, 16, 30, 32, 64, 80])
        norm_groups = rng.choice([g for g in (1, 2, 3, 4, heads) if (heads * vdim) % g == 0])
        right = _right(heads, vdim, rng.choice([4, 8, 18, 32, 64, 96]), groups, norm_groups, rng.choice([1, 2, 4, 4, 6]))
        if rng.random() < 0.3:
            if groups == 1:
                right.pop("groups")
            if norm_groups == 1:
                right.pop("norm_groups")
            if left["kv_heads"] == left["heads"]:
                left.pop("kv_heads")
            if left["vdim"] == left["dim"]:
                left.pop("vdim")
        layers.append(_parallel(left, right, ff))
    config = {"architecture": "Foduzen", "vocab": rng.choice([61, 128, 250]), "width": width,
              "norm": {"eps": rng.choice([1e-6, 1e-5, 3e-5])}, "initializer_range": 0.07, "layers": layers}
    if rng.random() < 0.8:
        config["embedding"] = {"scale": rng.choice([1.0, 4.0, 12.0])}
    return config


def make_model(folder: str, name: str) -> dict:
    """The folder through the package's random-weights mode; then the weights are moved to where a fault shows: the norms of q
    and k are raised (peaked attention weights: a wrong, missing or extra key changes the output), every norm weight and bias
    is spread, the convolutions' taps are of order one, the recurrences' decays reach from "forgets at once" to "keeps hundreds
    of tokens", their gates' matrices and the skip weights are raised, the activation's two numbers are of both signs.
    Returns {dir, config, weights (by checkpoint name, as stored), page_size, name}."""
    from safetensors.torch import load_file, save_file

    from lia_rs_b200.config import FoduzenConfig
    from lia_rs_b200.weights import write_random_model
    if name in FODUZEN:
        entry = FODUZEN[name]
    else:
        seed = int(name.split("-")[1])
        entry = dict(config=random_configuration(seed), seed=seed, page_size=(4, 8, 16)[seed % 3])
    write_random_model(FoduzenConfig.from_dict(entry["config"]), folder, seed=entry["seed"])
    path = os.path.join(folder, "model.safetensors")
    weights = load_file(path)
    g = torch.Generator().manual_seed(entry["seed"] + 100)
    bf16 = lambda t: t.to(torch.bfloat16)
    for key in list(weights):
        shape = weights[key].shape
        tail = key.split(".", 1)[1] if "." in key else key
        normal = lambda: torch.randn(shape, generator=g)
        if tail in ("mix.left.q.norm", "mix.left.k.norm"):
            weights[key] = bf16(1.8 + 0.4 * normal())
        elif tail == "mix.right.out" and entry.get("mute_right"):
            weights[key] = bf16(torch.zeros(shape))
        elif "norm" in tail or tail.endswith(".out"):
            weights[key] = bf16(1.0 + 0.3 * normal())
        elif tail.endswith("conv"):
            weights[key] = bf16(0.6 * normal())
        elif tail == "mix.lam":
            weights[key] = bf16(-4.0 + 4.0 * normal().clamp(-1.5, 1.5))
        elif tail == "mix.right.A_log":
            weights[key] = bf16(-3.0 + 2.5 * normal().clamp(-1.8, 1.8))
        elif tail == "mix.right.dt_bias":
            weights[key] = bf16(-0.5 + normal())
        elif tail in ("mix.right.D", "mlp.act"):
            weights[key] = bf16(normal())
        elif tail in ("mix.ra", "mix.ri"):
            weights[key] = bf16(2.0 * normal() / shape[-1] ** 0.5)
        elif tail.endswith(".b"):
            weights[key] = bf16(0.3 * normal())
    save_file(weights, path)
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    return dict(dir=folder, config=config, weights=weights, page_size=entry["page_size"], name=name)


_CACHE = {}


def plain_logits(model: dict, tokens) -> torch.Tensor:
    key = (model["name"], model["dir"], tuple(tokens))
    if key not in _CACHE:
        _CACHE[key] = plain_foduzen.forward(model["config"], model["weights"], list(tokens)).contiguous()
    return _CACHE[key]


def longest_sum(config: dict) -> int:
    sizes = [config["width"]]
    for layer in config["layers"]:
        m = layer["mixer"]
        if layer["type"] == "rglru":
            sizes.append(m["width"])
        else:
            sizes += [m["left"]["heads"] * max(m["left"]["dim"], m["left"].get("vdim", 0)),
                      m["right"]["heads"] * max(m["right"]["vdim"], m["right"]["state"])]
        if layer.get("mlp"):
            sizes.append(layer["mlp"]["ff"])
    return max(sizes)


def assert_close(actual, reference, dtype: str, what: str, config: dict):
    """Against the exact (64-bit) model.  32-bit: every logit within 8 K 2^-24 of the largest logit per layer that the sums
    pass through (K the model's longest sum; every layer has a recurrence, whose sums run along the sequence, and counts as
    four).  bfloat16: every row's root-mean-square error within 2.5e-2 of the largest logit, times the root of the number of
    layers (rounding noise of a layer adds to that of the layers before), and no single logit further off than three times
    that."""
    actual = torch.as_tensor(np.asarray(actual), dtype=torch.float64)
    reference = reference.to(torch.float64)
    assert actual.shape == reference.shape, f"{what}: shape {tuple(actual.shape)} vs {tuple(reference.shape)}"
    assert torch.isfinite(actual).all(), f"{what}: non-finite logits"
    layers = len(config["layers"])
    scale = max(1.0, float(reference.abs().max()))
    error = (actual - reference).abs()
    if dtype == "float32":
        limit = 8.0 * longest_sum(config) * 2.0 ** -24 * scale * 4 * layers
        worst = float(error.max())
    else:
        limit = 2.5e-2 * scale * layers ** 0.5
        worst = max(float((error ** 2).mean(dim=-1).sqrt().max()), float(error.max()) / 3.0)
    if worst > limit:
        row = int(error.max(dim=-1).values.argmax()) if error.dim() > 1 else 0
        raise AssertionError(f"{what}: error {worst:.3e} > {limit:.3e} (largest at wanted row {row})")
