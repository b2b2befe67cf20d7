"""The Botuvik configuration, its registration and the model description that is built from it, on the CPU: the round trip
through `to_dict`, refusals with the key's path, the order of layer runs, the parts chosen layer by layer with their
parameters, the tensor names and shapes, caches, states and junctions, random weights through the loader, and the plain
implementation's own consistency (portions of the recurrence, the order of runs)."""
import copy
import json
import os

import pytest
import torch

import botuvik_helpers as bh
import plain_botuvik as pb
from lia_rs_b200.config import BotuvikConfig, ConfigError, known_architectures, resolve_architecture
from lia_rs_b200.parts import KVCacheRequest

NAMES = list(bh.BOTUVIK)
F64 = torch.float64


def raw_config(name):
    return copy.deepcopy(bh.BOTUVIK[name]["config"])


@pytest.mark.parametrize("name", NAMES + ["random-7", "random-9"])
def test_round_trip_and_registry(name):
    raw = raw_config(name) if name in bh.BOTUVIK else bh.random_configuration(int(name.split("-")[1]))
    config = BotuvikConfig.from_dict(raw)
    again = BotuvikConfig.from_dict(config.to_dict())
    assert again == config and again.layers == config.layers and again.to_dict() == raw
    assert "Botuvik" in known_architectures() and resolve_architecture(raw).config_class is BotuvikConfig
    assert config.layer_runs() == pb.layer_order(raw)


def test_order_of_runs():
    raw = raw_config("bot-A")
    runs = BotuvikConfig.from_dict(raw).layer_runs()
    assert [layer for layer, _, _ in runs] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [t for _, t, _ in runs] == [None, 0, 0, 1, 1, 2, 2, None]
    assert [first for _, _, first in runs] == [False, True, False, True, False, True, False, False]
    raw.pop("loop")
    assert [layer for layer, _, _ in BotuvikConfig.from_dict(raw).layer_runs()] == [0, 1, 2, 3]


def test_refusals_name_the_key():
    good = raw_config("bot-A")

    def broken(change):
        raw = copy.deepcopy(good)
        change(raw)
        return raw
    moe = lambda r: r["layers"][0]["mlp"]
    cases = [
        (lambda r: r["layers"][0].update(type="mamba"), r"layers\[0\].type"),
        (lambda r: r["layers"][0]["mixer"].pop("gate_cap"), r"layers\[0\].mixer.gate_cap"),
        (lambda r: r["layers"][0]["mixer"].update(gate_cap=0), r"gate_cap"),
        (lambda r: r["layers"][0]["mixer"].pop("vdim"), r"layers\[0\].mixer.vdim"),
        (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
        (lambda r: r["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
        (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
        (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=40), "rot.dims"),
        (lambda r: r["layers"][1]["mixer"].pop("scale"), "mixer.scale"),
        (lambda r: moe(r).update(kind="glu"), "kind"),
        (lambda r: moe(r)["router"].update(top=7), "router.top"),
        (lambda r: moe(r)["router"]["groups"].update(count=4), "groups"),
        (lambda r: moe(r)["router"]["groups"].update(keep=4), "groups"),
        (lambda r: (moe(r)["router"].update(top=3), moe(r)["router"]["groups"].update(keep=1)), "kept groups"),
        (lambda r: moe(r)["shared"].update(ff=0), "shared.ff"),
        (lambda r: r["loop"].update(stop=5), "loop 1..5"),
        (lambda r: r["loop"].update(stop=1), "loop 1..1"),
        (lambda r: r["loop"].update(times=0), "loop.times"),
        (lambda r: r.pop("width"), "width"),
        (lambda r: r["norm"].pop("eps"), "norm.eps"),
        (lambda r: r.update(layers=[]), "non-empty"),
    ]
    for change, words in cases:
        with pytest.raises(ConfigError, match=words):
            BotuvikConfig.from_dict(broken(change))
    # sizes beyond the kernels are refused when the model is described, before any tensor is read
    architecture = resolve_architecture(good)
    for change, words in [(lambda r: r["layers"][0]["mixer"].update(dim=513), "head_dim"),
                          (lambda r: r["layers"][1]["mixer"].update(vdim=600), "v_head_dim"),
                          (lambda r: moe(r)["router"].update(experts=1500, groups=None), "experts")]:
        with pytest.raises(ValueError, match=words):
            architecture.build(BotuvikConfig.from_dict(broken(change)))


@pytest.mark.parametrize("name", NAMES)
def test_model_description(name):
    raw = raw_config(name)
    config = BotuvikConfig.from_dict(raw)
    spec = resolve_architecture(raw).build(config)
    width, order = raw["width"], pb.layer_order(raw)
    assert spec.max_positions is None and spec.position_table_name is None and spec.head_name == "head" and spec.streams == 1
    kinds = {"mlstm": "mlstm", "attention": "sink_attention"}
    assert [l.mixer.kind for l in spec.layers] == [kinds[l["type"]] for l in raw["layers"]]
    assert all(l.arrangement == "sandwich" for l in spec.layers)
    assert [l.feed_forward is None for l in spec.layers] == [l["mlp"] is None for l in raw["layers"]]
    assert [entry.layer for entry in spec.schedule] == [layer for layer, _, _ in order]
    names = {s.name: tuple(s.shape) for s in spec.tensor_specs() if not s.optional}
    assert names["embed"] == names["head"] == (raw["vocab"], width) and names["final.norm"] == (width,)
    if "loop" in raw:
        assert names["loop.step"] == (raw["loop"]["times"], width)
    else:
        assert "loop.step" not in names
    opens = {p: t for p, (_, t, first) in enumerate(order) if first}
    assert sorted(spec.junctions) == sorted(opens)
    for p, t in opens.items():
        assert spec.junctions[p].params["row"] == t and spec.junctions[p].params["first"] == (t > 0)
    caches, states = spec.cache_requests(), spec.state_requests()
    for p, (i, _, _) in enumerate(order):               # every run of a layer has a cache or a state of its own
        m = raw["layers"][i]["mixer"]
        if raw["layers"][i]["type"] == "attention":
            assert caches[p] == KVCacheRequest(m["kv_heads"], m["dim"], None, v_head_dim=m["vdim"]) and p not in states
        else:
            words = m["heads"] * (m["dim"] * m["vdim"] + m["dim"] + 1)
            assert p not in caches and states[p].dtype == torch.float32 and words <= states[p].shape[0] < words + 4
    for i, layer in enumerate(raw["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        assert names[p + "norm1"] == names[p + "norm1b"] == (width,)
        assert (p + "norm2" in names) == (p + "norm2b" in names) == (mlp is not None)
        if layer["type"] == "attention":
            assert names[p + "mix.sink"] == (m["heads"],) and names[p + "mix.q.b"] == (m["heads"] * m["dim"],)
            assert names[p + "mix.v"] == (m["kv_heads"] * m["vdim"], width) and names[p + "mix.o"] == (width, m["heads"] * m["vdim"])
            assert p + "mix.o.b" not in names and p + "mix.q.norm" not in names
        else:
            assert names[p + "mix.i"] == names[p + "mix.f"] == (m["heads"], width) and names[p + "mix.f.b"] == (m["heads"],)
            assert names[p + "mix.norm"] == (m["heads"] * m["vdim"],) and names[p + "mix.g"] == (m["heads"] * m["vdim"], width)
        if mlp and mlp["kind"] == "dense":
            assert names[p + "mlp.up"] == (mlp["ff"], width) and p + "mlp.gate" not in names
        elif mlp:
            experts = mlp["router"]["experts"]
            assert names[p + "mlp.router"] == (experts, width) and names[f"{p}mlp.e{experts - 1}.gate"] == (mlp["expert"]["ff"], width)
            assert f"{p}mlp.e{experts}.gate" not in names and p + "mlp.shared.sg" not in names and p + "mlp.correction" not in names
            assert ("shared" in mlp) == (p + "mlp.shared.up" in names)


@pytest.mark.parametrize("name", NAMES)
def test_random_weights_load(tmp_path, name):
    from lia_rs_b200.weights import WeightError, load_weights
    model = bh.make_model(str(tmp_path / "m"), name)
    spec = resolve_architecture(model["config"]).build(BotuvikConfig.from_dict(model["config"]))
    loaded = load_weights(model["dir"], spec.tensor_specs())
    assert set(loaded) == set(model["weights"])
    for key, tensor in loaded.items():
        assert torch.equal(tensor, model["weights"][key]), key
    with open(os.path.join(model["dir"], "config.json")) as f:
        raw = json.load(f)
    raw["layers"][0]["mlp"] = {"kind": "dense", "ff": 12}           # other sizes than the stored tensors'
    with pytest.raises(WeightError, match=r"l0.mlp.up"):
        load_weights(model["dir"], resolve_architecture(raw).build(BotuvikConfig.from_dict(raw)).tensor_specs())


def test_absent_keys_have_their_defaults():
    raw = raw_config("bot-E")
    raw["layers"][0]["mixer"] = {"heads": 6, "dim": 24, "scale": 0.2}
    raw["layers"][1]["mlp"]["router"].pop("groups")
    raw["layers"][1]["mlp"].pop("shared")
    raw.pop("loop")
    spec = resolve_architecture(raw).build(BotuvikConfig.from_dict(raw))
    params = spec.layers[0].mixer.params
    assert params["kv_heads"] == 6 and params["v_head_dim"] == 24 and params["softcap"] is None and params["rot"] is None
    assert spec.layers[1].feed_forward.params["groups"] is None and spec.layers[1].feed_forward.params["shared"] is None
    assert not spec.junctions


def test_the_plain_recurrence_in_portions():
    """Cut anywhere and carried on from its state the plain recurrence is the whole one; its maximum starts at zero."""
    g = torch.Generator().manual_seed(3)
    T, H, d, dv = 40, 2, 6, 5
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (d, d, dv))
    i = 3 * torch.randn(T, H, generator=g, dtype=F64)
    f = torch.nn.functional.logsigmoid(2 + 2 * torch.randn(T, H, generator=g, dtype=F64))
    whole, end = pb.mlstm_recurrence(q, k, v, i, f)
    parts, state = [], None
    for a, b in ((0, 1), (1, 3), (3, 20), (20, 40)):
        out, state = pb.mlstm_recurrence(q[a:b], k[a:b], v[a:b], i[a:b], f[a:b], state)
        parts.append(out)
    assert torch.allclose(torch.cat(parts), whole, atol=1e-12) and all(torch.allclose(x, y) for x, y in zip(state, end))
    # without the running maximum: S_t = sum_j exp(F_t - F_j + i_j) k_j v_j^T
    F = torch.cumsum(f, 0)
    t = T - 1
    weight = torch.exp(F[t] - F + i)
    S = torch.einsum("jh,jhd,jhe->hde", weight, k, v)
    n = torch.einsum("jh,jhd->hd", weight, k)
    m = torch.maximum(F[t], (F[t] - F + i).max(dim=0).values)         # the start counts as a gate of zero
    below = torch.maximum((n * q[t]).sum(-1).abs() * torch.exp(-m), torch.exp(-m)) + 1e-6
    assert torch.allclose(torch.einsum("hde,hd->he", S, q[t]) * torch.exp(-m)[:, None] / below[:, None], whole[t], atol=1e-10)


def test_a_sink_and_a_cap_together_are_taken():
    from lia_rs_b200.parts.softmax_attention import SinkAttention
    params = resolve_architecture(raw_config("bot-E")).build(BotuvikConfig.from_dict(raw_config("bot-E"))).layers[0].mixer.params
    SinkAttention.check_params(params)
    with pytest.raises(ValueError, match="sink"):
        SinkAttention.check_params({**params, "sink": "some"})
    with pytest.raises(ValueError, match="qk_norm"):
        SinkAttention.check_params({**params, "qk_norm": "ahead"})
