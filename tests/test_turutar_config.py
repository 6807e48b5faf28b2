"""The Turutar configuration, its plan and tensor names, and the plain implementation against closed
forms.  All on the CPU."""

import copy
import math

import pytest
import torch

import turutar_tiny as tiny
from plain import turutar_plain as plain

from thing_htn_2026_b200.config import ConfigError, config_from_dict, named_config_json, named_configs
from thing_htn_2026_b200.config.base import looped_schedule
from thing_htn_2026_b200.models.decoder import tensor_specs_of_plan
from thing_htn_2026_b200.weights.loader import merge_specs


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_reading_and_writing_back(name):
    data = tiny.config_json(name)
    config = config_from_dict(data)
    assert config.architecture == "Turutar"
    assert config.to_dict() == data
    assert config_from_dict(config.to_dict()) == config


def test_named_configurations_are_read():
    names = [n for n in named_configs() if n.startswith("turutar-")]
    assert len(names) >= 3
    for name in names:
        assert config_from_dict(named_config_json(name)).architecture == "Turutar"


def test_a_looped_schedule():
    runs = lambda *args: [(e.layer, e.adds_start) for e in looped_schedule(*args)]
    assert runs(3) == [(0, False), (1, False), (2, False)]
    assert runs(4, 1, 3, 3) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert runs(2, 0, 2, 1) == [(0, False), (1, False)]
    assert runs(3, 2, 3, 2) == [(0, False), (1, False), (2, False), (2, True)]
    schedule = looped_schedule(4, 0, 4, 2)
    assert [e.cache for e in schedule] == list(range(8)) and all(e.writes_cache for e in schedule)


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_the_plan_runs_layers_in_the_order_of_the_plain_implementation(name):
    data = tiny.config_json(name)
    plan = config_from_dict(data).plan()
    assert [(e.layer, e.adds_start) for e in plan.schedule] == plain.layer_runs(data)
    assert plan.n_cache_entries == len(plan.schedule)


def test_the_plan_names_parts_and_their_constants():
    plan = config_from_dict(tiny.config_json("a")).plan()
    assert [layer.block.kind for layer in plan.layers] == ["parallel"] * 3
    block = plan.layers[0].block
    assert block.params["layer_scale"] and dict(block.tensors) == {"mixer_scale": "l0.ls1", "ffn_scale": "l0.ls2"}
    assert block.params["norm"].params["gain_offset"] == 1.0
    mixer = block.params["mixer"].params
    assert mixer["window"] == 20 and mixer["sinks"] == 0.0 and mixer["gate"] == "head" and mixer["values"] == "keys"
    assert mixer["qk_norm_scope"] == "projection" and mixer["position"] is None and mixer["biases"] == ("q", "k")
    assert block.params["ffn"].params["limit"] == 0.6 and block.params["ffn"].params["slope"] == 1.702
    lat = plan.layers[1].block.params["mixer"].params
    assert lat["q_rank"] == 14 and lat["latent_rank"] == 22 and lat["sinks"] == "learned" and lat["gate_scope"] == "head"
    assert lat["position"].params["layout"] == "interleaved" and lat["position"].params["theta"] == 10000.0
    side = plan.layers[2].block.params["side"].params
    assert side["column"] == 20 and side["dim"] == 10 and side["table_width"] == 30
    assert side["norm"].params["gain_offset"] == 0.0
    assert plan.layers[2].block.params.get("ffn") is None and dict(plan.layers[2].block.tensors) == {"mixer_scale": "l2.ls1"}
    assert plan.embedding.params["norm"].tensors["weight"] == "embed.norm"
    other = config_from_dict(tiny.config_json("c")).plan()
    assert other.layers[0].block.params.get("side") is None and other.layers[0].block.params["mixer"].params["position"] is None
    assert other.layers[2].block.params["mixer"].params["window"] is None


def test_tensor_names_and_shapes():
    specs = merge_specs(tensor_specs_of_plan(config_from_dict(tiny.config_json("a")).plan()))
    shape = {name: spec.shape for name, spec in specs.items()}
    assert shape["embed"] == (200, 48) and shape["embed.norm"] == (48,) and shape["head"] == (200, 48) and shape["final.norm"] == (48,)
    assert shape["side.embed"] == (200, 30) and shape["l1.side.gate"] == (10, 48) and shape["l1.side.proj"] == (48, 10)
    assert shape["l1.side.norm"] == (48,) and shape["l0.ls1"] == (48,) and shape["l0.ls2"] == (48,) and "l2.ls2" not in shape
    assert shape["l0.mix.q"] == (48, 48) and shape["l0.mix.q.b"] == (48,) and shape["l0.mix.k"] == (24, 48) and shape["l0.mix.k.b"] == (24,)
    assert shape["l0.mix.q.norm"] == (48,) and shape["l0.mix.k.norm"] == (24,) and shape["l0.mix.g"] == (4, 48) and shape["l0.mix.o"] == (48, 48)
    assert "l0.mix.v" not in shape and "l0.mix.sink" not in shape
    assert shape["l1.mix.dq"] == (14, 48) and shape["l1.mix.dq.norm"] == (14,) and shape["l1.mix.uq"] == (48, 14)
    assert shape["l1.mix.dkv"] == (28, 48) and shape["l1.mix.dkv.norm"] == (22,) and shape["l1.mix.uk"] == (30, 22)
    assert shape["l1.mix.uv"] == (60, 22) and shape["l1.mix.sink"] == (3,) and shape["l1.mix.g"] == (3, 48) and shape["l1.mix.o"] == (48, 60)
    assert shape["l0.mlp.gate"] == (40, 48) and shape["l0.mlp.down"] == (48, 40) and "l2.mlp.up" not in shape
    assert "side.embed" not in merge_specs(tensor_specs_of_plan(config_from_dict(tiny.config_json("c")).plan()))


@pytest.mark.parametrize("change, key", [
    (lambda d: d["layers"][0].__setitem__("type", "wkv"), "type"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("vdim", 8), "vdim"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("rot", {"base": 10.0, "dims": 2}), "rot"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("dims", 4), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("mask", {"size": 8}), "mask"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["loop"].__setitem__("stop", 4), "loop"),
    (lambda d: d["loop"].__setitem__("stop", 1), "loop"),
    (lambda d: d["loop"].__setitem__("times", 0), "times"),
    (lambda d: d["token_side"].__setitem__("dim", 0), "dim"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_what_cannot_run_is_refused_with_its_key(change, key):
    data = copy.deepcopy(tiny.config_json("a"))
    change(data)
    with pytest.raises(ConfigError) as info:
        config_from_dict(data)
    assert key in str(info.value)


# ----------------------------------------------------------------------------- the plain implementation against closed forms

EXACT = plain.Arithmetic(torch.float64)


def test_the_norms_and_the_embedding():
    x = torch.tensor([[3.0, 4.0]]).double()
    assert torch.allclose(plain.norm_around_zero(x, torch.tensor([0.0, 1.0]).double(), 0.5), torch.tensor([[3.0, 8.0]]).double() / math.sqrt(13.0))
    w = {"embed": torch.tensor([[1.0, 1.0], [3.0, 4.0]]), "embed.norm": torch.tensor([0.0, 1.0])}
    got = plain.embed(w, {"norm": {"eps": 0.5}}, torch.tensor([1, 0]), torch.float64)
    assert torch.allclose(got, torch.tensor([[3.0 / math.sqrt(13.0), 8.0 / math.sqrt(13.0)],
                                             [1.0 / math.sqrt(1.5), 2.0 / math.sqrt(1.5)]]).double())


def test_an_extra_term_takes_weight_and_brings_nothing():
    score = torch.tensor([[0.0, math.log(2.0), 50.0]]).double()
    visible = torch.tensor([[True, True, False]])
    got = plain.softmax_with_extra(score, visible, torch.tensor(0.0).double())
    assert torch.allclose(got, torch.tensor([[0.25, 0.5, 0.0]]).double())
    got = plain.softmax_with_extra(score, visible, torch.tensor(math.log(7.0)).double())
    assert torch.allclose(got, torch.tensor([[0.1, 0.2, 0.0]]).double())
    assert plain.softmax_with_extra(score - 800.0, visible, torch.tensor(0.0).double()).abs().max() == 0.0


def test_windowed_attention_by_hand():
    """Scores of zero (no scale to speak of): a row's weights are one over its window's tokens and the extra
    one; the values are the keys with their bias, before the norm; the gate is one number per head."""
    T, H, d, W = 7, 2, 3, 3
    m = {"heads": H, "kv_heads": 1, "dim": d, "scale": 1e-30, "mask": {"size": W}}
    g = torch.Generator().manual_seed(3)
    w = {"x." + k: torch.randn(*s, generator=g).double() for k, s in
         {"q": (6, 5), "q.b": (6,), "k": (3, 5), "k.b": (3,), "q.norm": (6,), "k.norm": (3,), "g": (2, 5), "o": (6, 6)}.items()}
    w["x.o"] = torch.eye(6).double()
    h = torch.randn(T, 5, generator=g).double()
    out = plain.window_attention(EXACT, h, w, "x.", m, 1e-6).reshape(T, H, d)
    v = h @ w["x.k"].t() + w["x.k.b"]
    gate = torch.sigmoid(h @ w["x.g"].t())
    for t in range(T):
        seen = v[max(0, t - W + 1):t + 1]
        assert torch.allclose(out[t], gate[t][:, None] * (seen.sum(0) / (1 + len(seen)))[None])


def test_latent_attention_of_a_single_token_shares_with_its_sink():
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "q_rank": 3, "kv_rank": 5, "scale": 0.7, "rot": {"base": 10.0, "dims": 2}}
    g = torch.Generator().manual_seed(3)
    w = {"x." + k: torch.randn(*s, generator=g).double() for k, s in
         {"dq": (3, 6), "dq.norm": (3,), "uq": (10, 3), "dkv": (7, 6), "dkv.norm": (5,), "uk": (6, 5), "uv": (8, 5), "sink": (2,),
          "g": (2, 6), "o": (6, 8)}.items()}
    h = torch.randn(1, 6, generator=g).double()
    out = plain.latent_attention(EXACT, h, w, "x.", m, 1e-6)
    down = (h @ w["x.dkv"].t())[0]
    c = plain.rms_divide(down[:5], 1e-6) * w["x.dkv.norm"]
    q = (w["x.uq"] @ (plain.rms_divide(w["x.dq"] @ h[0], 1e-6) * w["x.dq.norm"])).reshape(2, 5)
    k = torch.cat([(w["x.uk"] @ c).reshape(2, 3), down[5:].expand(2, 2)], dim=1)
    s = (q * k).sum(1) * 0.7
    share = torch.exp(s) / (torch.exp(s) + torch.exp(w["x.sink"]))
    v = (w["x.uv"] @ c).reshape(2, 4) * (share * torch.sigmoid(w["x.g"] @ h[0]))[:, None]
    assert torch.allclose(out, v.reshape(1, 8) @ w["x.o"].t(), atol=1e-12)


def test_the_rotation_turns_neighbours():
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0]]).double()
    got = plain.rotate_neighbours(x, torch.tensor([3]), 100.0)
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    assert torch.allclose(got, torch.tensor([[math.cos(a), math.sin(a), -2.0 * math.sin(b), 2.0 * math.cos(b)]]).double())


def test_the_feed_forward_clamps_its_gate_from_above_and_its_up_from_both_sides():
    w = {"m.gate": torch.tensor([[1.0], [1.0], [1.0]]).double(), "m.up": torch.tensor([[1.0], [-1.0], [0.1]]).double(),
         "m.down": torch.eye(3).double()}
    f = lambda g, u: g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0)
    got = plain.clamped_feed_forward(EXACT, torch.tensor([[5.0], [-5.0]]).double(), w, "m.", 2.0)
    assert torch.allclose(got, torch.tensor([[f(2.0, 2.0), f(2.0, -2.0), f(2.0, 0.5)], [f(-5.0, -2.0), f(-5.0, 2.0), f(-5.0, -0.5)]]).double())


def test_the_token_part_takes_its_layers_columns_and_its_own_norm():
    w = {"side.embed": torch.tensor([[1.0, 2.0, 3.0, 4.0], [5.0, 6.0, 7.0, 8.0]]), "l1.side.gate": torch.eye(2), "l1.side.proj": torch.eye(2),
         "l1.side.norm": torch.tensor([1.0, 10.0])}
    x = torch.tensor([[0.5, -1.0]]).double()
    gelu = torch.nn.functional.gelu(x, approximate="tanh")[0]
    y = gelu * torch.tensor([7.0, 8.0]).double()
    want = y / torch.sqrt((y * y).mean() + 0.25) * torch.tensor([1.0, 10.0]).double()
    assert torch.allclose(plain.token_side(EXACT, x, torch.tensor([1]), w, 1, 2, 0.25)[0], want)


def test_a_later_pass_adds_the_start_once():
    """Layers that add nothing (zero scales, a zero norm on the token part): after three passes the stream
    is three times its start."""
    data = tiny.config_json("b")
    from thing_htn_2026_b200.weights import random_tensors_cpu
    w = {k: v.float() for k, v in random_tensors_cpu(config_from_dict(data), 1).items()}
    for key in w:
        if key.endswith((".ls1", ".ls2", "side.norm")):
            w[key] = torch.zeros_like(w[key])
    toks = tiny.tokens("b", 9, 1)
    start = plain.embed(w, data, torch.tensor(toks), torch.float64)
    after = plain.model_forward(None, toks, torch.float64, (data, w))[1]
    assert [round((a / start).mean().item(), 9) for a in after] == [1.0, 1.0, 2.0, 2.0, 3.0, 3.0, 3.0]


# ----------------------------------------------------------------------------- what comparisons with it show


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    return tiny.write_model(str(tmp_path_factory.mktemp("turutar") / "a"), "a")


def changed(folder, change):
    """Exact logits of 150 tokens with a mistake planted in the plain implementation, and without."""
    config, w = plain.read_model(folder)
    toks = tiny.tokens("a", 150, 77)
    right = plain.model_forward(None, toks, torch.float64, (config, w))[0].numpy()
    change(config, w)
    difference = plain.model_forward(None, toks, torch.float64, (config, w))[0].numpy() - right
    return (difference - difference.mean(axis=1, keepdims=True)).std(axis=1)


@pytest.mark.parametrize("what, change", [
    ("window one longer", lambda c, w: c["layers"][0]["mixer"]["mask"].update(size=21)),
    ("window one shorter", lambda c, w: c["layers"][2]["mixer"]["mask"].update(size=32)),
    ("sinks left out", lambda c, w: w.update({"l1.mix.sink": torch.full((3,), -100.0)})),
    ("biases left out", lambda c, w: w.update({"l0.mix.k.b": torch.zeros(24)})),
    ("one pass fewer", lambda c, w: c["loop"].update(times=1)),
    ("loop from the first layer", lambda c, w: c["loop"].update(start=0)),
    ("another layer's columns", lambda c, w: w.update({"side.embed": w["side.embed"].roll(10, 1)})),
    ("layer scales swapped", lambda c, w: w.update({"l0.ls1": w["l0.ls2"], "l0.ls2": w["l0.ls1"]})),
    ("gate of another head", lambda c, w: w.update({"l0.mix.g": w["l0.mix.g"].roll(1, 0)})),
    ("another limit", lambda c, w: c["layers"][0]["mlp"].update(limit=0.7)),
])
def test_what_the_comparisons_would_show(folder, what, change):
    """Mistakes planted in the plain implementation move the logits far beyond the tolerances of the comparisons on the device."""
    assert changed(folder, change)[60:].max() > 1e-2, what
