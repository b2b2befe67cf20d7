"""The Foduzen configuration, its registration and the model description that is built from it, on the CPU: the round trip
through `to_dict`, refusals with the key's path, the parts chosen layer by layer with their parameters, the tensor names and
shapes, caches and states, and random weights through the loader."""
import copy
import json
import os

import pytest
import torch

import foduzen_helpers as fh
from lia_rs_b200.config import ConfigError, FoduzenConfig, known_architectures, resolve_architecture
from lia_rs_b200.parts import KVCacheRequest

NAMES = list(fh.FODUZEN)


def raw_config(name):
    return copy.deepcopy(fh.FODUZEN[name]["config"])


@pytest.mark.parametrize("name", NAMES + ["random-7", "random-9"])
def test_round_trip_and_registry(name):
    raw = raw_config(name) if name in fh.FODUZEN else fh.random_configuration(int(name.split("-")[1]))
    config = FoduzenConfig.from_dict(raw)
    again = FoduzenConfig.from_dict(config.to_dict())
    assert again == config and again.layers == config.layers
    assert "Foduzen" in known_architectures() and resolve_architecture(raw).config_class is FoduzenConfig
    assert config.embedding_scale == (raw.get("embedding") or {}).get("scale", 1.0)


def test_refusals_name_the_key():
    good = raw_config("fod-A")

    def broken(change):
        raw = copy.deepcopy(good)
        change(raw)
        return raw
    cases = [
        (lambda r: r["layers"][0].update(type="mamba"), r"layers\[0\].type"),
        (lambda r: r["layers"][0]["mixer"].update(blocks=5), "multiple of blocks"),
        (lambda r: r["layers"][0]["mixer"].update(conv=0), r"layers\[0\].mixer.conv"),
        (lambda r: r["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple of kv_heads"),
        (lambda r: r["layers"][1]["mixer"]["left"]["mask"].update(size=0), r"left.mask.size"),
        (lambda r: r["layers"][1]["mixer"]["left"].pop("scale"), r"left.scale"),
        (lambda r: r["layers"][1]["mixer"]["right"].update(groups=3), "multiple of groups"),
        (lambda r: r["layers"][1]["mixer"]["right"].update(norm_groups=5), "multiple of norm_groups"),
        (lambda r: r["layers"][1]["mixer"]["right"].pop("state"), r"right.state"),
        (lambda r: r["layers"][1]["mixer"].pop("right"), "'right'"),
        (lambda r: r["layers"][1]["mlp"].update(kind="glu"), "kind"),
        (lambda r: r.pop("width"), "width"),
        (lambda r: r["norm"].pop("eps"), "norm.eps"),
        (lambda r: r.update(layers=[]), "non-empty"),
    ]
    for change, words in cases:
        with pytest.raises(ConfigError, match=words):
            FoduzenConfig.from_dict(broken(change))
    # sizes beyond the kernels are refused when the model is described, before any tensor is read
    architecture = resolve_architecture(good)
    for change, words in [(lambda r: r["layers"][0]["mixer"].update(conv=9), "taps"),
                          (lambda r: r["layers"][1]["mixer"]["right"].update(state=300), "state"),
                          (lambda r: r["layers"][1]["mixer"]["left"].update(vdim=600), "v_head_dim")]:
        with pytest.raises(ValueError, match=words):
            architecture.build(FoduzenConfig.from_dict(broken(change)))


@pytest.mark.parametrize("name", NAMES)
def test_model_description(name):
    raw = raw_config(name)
    config = FoduzenConfig.from_dict(raw)
    spec = resolve_architecture(raw).build(config)
    width = raw["width"]
    assert spec.max_positions is None and spec.position_table_name is None and spec.head_name == "head"
    assert spec.sinusoidal_base == 10000.0 and spec.streams == 1 and spec.logit_scale == 1.0
    assert spec.embedding_scale == config.embedding_scale
    kinds = {"rglru": "rglru", "parallel": "side_by_side"}
    assert [l.mixer.kind for l in spec.layers] == [kinds[l["type"]] for l in raw["layers"]]
    assert all(l.arrangement == "postnorm" and l.norm.params["single"] for l in spec.layers)
    assert [l.feed_forward is None for l in spec.layers] == [l["mlp"] is None for l in raw["layers"]]
    names = {s.name: tuple(s.shape) for s in spec.tensor_specs() if not s.optional}
    assert names["embed"] == names["head"] == (raw["vocab"], width) and names["final.norm"] == ()
    caches, states = spec.cache_requests(), spec.state_requests()
    assert sorted(states) == list(range(len(raw["layers"])))
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        assert names[p + "norm1"] == () and (p + "norm2" in names) == (layer["mlp"] is not None)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            assert names[p + "mlp.up"] == (ff, width) and names[p + "mlp.down"] == (width, ff) and names[p + "mlp.act"] == (2,)
        if layer["type"] == "rglru":
            size = m["width"] // m["blocks"]
            assert names[p + "mix.ra"] == (m["blocks"], size, size) and names[p + "mix.ra.b"] == (m["blocks"], size)
            assert names[p + "mix.conv"] == (m["width"], m["conv"]) and names[p + "mix.lam"] == (m["width"],)
            assert i not in caches
            ring = m["conv"] * m["width"] if m["conv"] > 1 else 0
            assert states[i].dtype == torch.float32 and ring + m["width"] <= states[i].shape[0] < ring + m["width"] + 8
        else:
            left, right = m["left"], m["right"]
            window = left["mask"]["size"] if "mask" in left else None
            assert caches[i] == KVCacheRequest(left["kv_heads"], left["dim"], window, v_head_dim=left["vdim"])
            inner, conv = right["heads"] * right["vdim"], right["heads"] * right["vdim"] + 2 * right["groups"] * right["state"]
            assert names[p + "mix.right.in"] == (inner + conv + right["heads"], width)
            assert names[p + "mix.right.conv"] == (conv, right["conv"]) and names[p + "mix.right.norm"] == (inner,)
            assert names[p + "mix.left.g"] == (left["heads"] * left["vdim"], width) and names[p + "mix.left.o.b"] == (width,)
            assert names[p + "mix.left.q.norm"] == (left["dim"],)
            assert names[p + "mix.left.out"] == names[p + "mix.right.out"] == (width,)


@pytest.mark.parametrize("name", NAMES)
def test_random_weights_load(tmp_path, name):
    from lia_rs_b200.weights import WeightError, load_weights
    model = fh.make_model(str(tmp_path / "m"), name)
    spec = resolve_architecture(model["config"]).build(FoduzenConfig.from_dict(model["config"]))
    loaded = load_weights(model["dir"], spec.tensor_specs())
    assert set(loaded) == set(model["weights"])
    for key, tensor in loaded.items():
        assert torch.equal(tensor, model["weights"][key]), key
    with open(os.path.join(model["dir"], "config.json")) as f:
        raw = json.load(f)
    raw["layers"][0]["mlp"] = {"kind": "dense", "ff": 12}           # other sizes than the stored tensors'
    with pytest.raises(WeightError, match=r"l0.mlp.up"):
        load_weights(model["dir"], resolve_architecture(raw).build(FoduzenConfig.from_dict(raw)).tensor_specs())


def test_absent_keys_have_their_defaults():
    raw = raw_config("fod-B")
    layer = raw["layers"][0]["mixer"]
    layer["left"].pop("vdim")
    layer["left"].pop("kv_heads")
    layer["right"].pop("groups")
    layer["right"].pop("norm_groups")
    spec = resolve_architecture(raw).build(FoduzenConfig.from_dict(raw))
    left, right = (m["params"] for m in spec.layers[0].mixer.params["members"])
    assert left["kv_heads"] == left["heads"] and left["v_head_dim"] == left["head_dim"] and left["window"] is None
    assert right["groups"] == right["norm_groups"] == 1
    assert [m["scale"] for m in spec.layers[0].mixer.params["members"]] == [0.5, 0.5]
    assert spec.embedding_scale == 1.0


def test_arrangements_that_cannot_norm_a_sum_refuse_it():
    """A mixer that leaves a sum of terms fits only an arrangement that norms its sublayers' outputs; norms for some members
    only are refused."""
    from lia_rs_b200.parts.side_by_side import SideBySide
    spec = resolve_architecture(raw_config("fod-A")).build(FoduzenConfig.from_dict(raw_config("fod-A")))
    params = copy.deepcopy(spec.layers[1].mixer.params)
    SideBySide.check_params(params)
    params["members"][0].pop("norm")
    with pytest.raises(ValueError, match="norms for all members"):
        SideBySide.check_params(params)
