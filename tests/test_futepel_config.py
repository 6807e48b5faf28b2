"""The Futepel configuration, its plan and tensor names, and the plain implementation against closed
forms.  All on the CPU."""

import copy
import math

import pytest
import torch

import futepel_tiny as tiny
from plain import futepel_plain as plain

from thing_htn_2026_b200.config import ConfigError, config_from_dict, named_config_json, named_configs
from thing_htn_2026_b200.models.decoder import tensor_specs_of_plan
from thing_htn_2026_b200.weights.loader import check_names, merge_specs


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_reading_and_writing_back(name):
    data = tiny.config_json(name)
    config = config_from_dict(data)
    assert config.architecture == "Futepel"
    assert config.to_dict() == data
    assert config_from_dict(config.to_dict()) == config


def test_named_configurations_are_read():
    names = [n for n in named_configs() if n.startswith("futepel-")]
    assert len(names) >= 3
    for name in names:
        assert config_from_dict(named_config_json(name)).architecture == "Futepel"


def test_the_plan_names_parts_and_their_constants():
    plan = config_from_dict(tiny.config_json("b")).plan()
    assert [layer.block.kind for layer in plan.layers] == ["pre_norm"] * 3
    assert [layer.block.params["mixer"].kind for layer in plan.layers] == ["state_space", "latent_attention", "time_mixing"]
    attention = plan.layers[1].block.params["mixer"].params
    assert attention["gate_scope"] == "head" and attention["gated"] and attention["softmax_weights"] == "float32"
    rope = attention["position"].params
    assert rope["layout"] == "half" and rope["rotary_dim"] == 16 and rope["theta"] == 500.0
    assert dict(rope["scaling"]) == {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 1.0}
    assert plan.layers[1].block.params["ffn"].kind == "routed_glu_experts"
    assert plan.layers[2].block.params.get("ffn") is None
    assert plan.embedding.params["positions"] == {"kind": "learned", "size": 256}
    assert plan.embedding.params["pairs"] == {"buckets": 500, "mul_before": 3, "mul_token": 1000003}
    assert plan.max_positions == 256
    other = config_from_dict(tiny.config_json("c")).plan()
    assert other.embedding.params.get("pairs") is None and "pairs" not in other.embedding.tensors
    assert other.layers[0].block.params["mixer"].params["position"] is None
    assert other.layers[2].block.params["ffn"].kind == "squared_relu"


def test_tensor_names_and_shapes():
    specs = merge_specs(tensor_specs_of_plan(config_from_dict(tiny.config_json("a")).plan()))
    shape = {name: spec.shape for name, spec in specs.items()}
    assert shape["embed"] == (200, 48) and shape["head"] == (200, 48) and shape["final.norm"] == (48,)
    assert shape["bigram"] == (32, 48) and shape["pos"] == (300, 48) and shape["l0.norm1"] == (48,)
    assert shape["l0.mix.mu.w"] == (48,) and shape["l0.mix.r"] == (30, 48) and shape["l0.mix.w1"] == (5, 48)
    assert shape["l0.mix.w2"] == (30, 5) and shape["l0.mix.w0"] == (30,) and shape["l0.mix.u"] == (3, 10)
    assert shape["l0.mix.norm"] == (30,) and shape["l0.mix.o"] == (48, 30)
    assert shape["l1.mix.q"] == (48, 48) and shape["l1.mix.dkv"] == (28, 48) and shape["l1.mix.dkv.norm"] == (22,)
    assert shape["l1.mix.uk"] == (30, 22) and shape["l1.mix.uv"] == (60, 22) and shape["l1.mix.g"] == (3, 48)
    assert shape["l1.mlp.up"] == (56, 48) and shape["l1.mlp.down"] == (48, 56) and "l1.mlp.router" not in shape
    assert shape["l2.mix.in"] == (2 * 30 + 2 * 21 + 6, 48) and shape["l2.mix.conv"] == (72, 4) and shape["l2.mix.conv.b"] == (72,)
    assert shape["l2.mix.A_log"] == (6,) and shape["l2.mix.D"] == (6,) and shape["l2.mix.norm"] == (30,)
    assert "l2.norm2" not in shape and "l2.mlp.up" not in shape
    assert shape["l0.mlp.e4.gate"] == (24, 48) and shape["l0.mlp.shared.down"] == (48, 40) and "l4.mlp.shared.up" not in shape
    assert "bigram" not in merge_specs(tensor_specs_of_plan(config_from_dict(tiny.config_json("c")).plan()))


def test_a_rank_that_only_the_checkpoint_gives():
    data = tiny.config_json("a")
    data = copy.deepcopy(data)
    del data["layers"][0]["mixer"]["rank"]
    specs = merge_specs(tensor_specs_of_plan(config_from_dict(data).plan()))
    assert specs["l0.mix.w1"].shape == (-1, 48) and specs["l0.mix.w2"].shape == (30, -1)
    found = {name: spec.shape for name, spec in specs.items()}
    found["l0.mix.w1"], found["l0.mix.w2"] = (9, 48), (30, 9)
    assert check_names("x", specs, found, strict=True) == []


@pytest.mark.parametrize("change, key", [
    (lambda d: d["layers"][0].__setitem__("type", "attention"), "type"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("dim", 0), "dim"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("dims", 4), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("scaling", {"factor": 2.0}), "original"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("window", 8), "window"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][2]["mixer"].__setitem__("groups", 4), "groups"),
    (lambda d: d["layers"][2]["mixer"].__setitem__("norm_groups", 7), "norm_groups"),
    (lambda d: d["layers"][0]["mlp"]["router"].__setitem__("top", 6), "top"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "glu"), "kind"),
    (lambda d: d["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda d: d["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda d: d.pop("max_positions"), "max_positions"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_what_cannot_run_is_refused_with_its_key(change, key):
    data = copy.deepcopy(tiny.config_json("a"))
    change(data)
    with pytest.raises(ConfigError) as info:
        config_from_dict(data)
    assert key in str(info.value)


# ----------------------------------------------------------------------------- the plain implementation against closed forms


def test_the_embedding_adds_a_pair_and_a_place():
    w = {"embed": torch.tensor([[1.0], [2.0], [3.0]]), "bigram": torch.tensor([[10.0], [20.0], [30.0], [40.0], [50.0], [60.0]]),
         "pos": torch.tensor([[0.1], [0.2], [0.3], [0.4]])}
    config = {"embedding": {"scale": 2.0, "bigram": {"buckets": 5, "mul_prev": 2, "mul_cur": 3}}}
    got = plain.embed(w, config, torch.tensor([1, 2, 0, 0]), torch.float64)
    # rows: the last one, (2 + 6) % 5 = 3, (4 + 0) % 5 = 4, 0
    assert torch.allclose(got[:, 0], torch.tensor([4.0 + 60.0 + 0.1, 6.0 + 40.0 + 0.2, 2.0 + 50.0 + 0.3, 2.0 + 10.0 + 0.4]).double(),
                          atol=1e-6)


def test_scaled_frequencies_keep_the_fast_pairs_and_stretch_the_slow_ones():
    freq, magnitude = plain.yarn_frequencies({"base": 10000.0, "dims": 32,
                                              "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}})
    plain_freq, one = plain.yarn_frequencies({"base": 10000.0, "dims": 32})
    assert one == 1.0 and abs(magnitude - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    assert freq[0] == plain_freq[0] and abs(freq[-1] - plain_freq[-1] / 8.0) < 1e-18
    assert all(a >= b * (1 - 1e-12) for a, b in zip(freq, freq[1:]))
    # pair (i, i + half) turns by position times frequency, lengths grow by the magnitude
    x = torch.zeros(1, 1, 4, dtype=torch.float64)
    x[0, 0, 0] = 1.0
    turned = plain.rotate(x, torch.tensor([2]), {"base": 10000.0, "dims": 4})
    assert torch.allclose(turned[0, 0], torch.tensor([math.cos(2.0), 0.0, math.sin(2.0), 0.0]).double())


def test_time_mixing_by_hand():
    """Two tokens, one head of one entry: the second token sees the first through the decayed state, its
    own product through the bonus only, and every projection its own blend of the two."""
    m = {"heads": 1, "dim": 1}
    mu = dict(r=0.0, k=0.25, v=0.5, g=0.0, w=1.0)
    w = {f"x.mu.{s}": torch.tensor([v]).double() for s, v in mu.items()}
    w.update({f"x.{s}": torch.ones(1, 1).double() for s in ("r", "k", "v", "g", "w1", "w2", "o")})
    w.update({"x.w0": torch.tensor([-1.0]).double(), "x.u": torch.tensor([[3.0]]).double(), "x.norm": torch.ones(1).double()})
    h = torch.tensor([[2.0], [4.0]]).double()
    out = plain.time_mixing(plain.Arithmetic(torch.float64), h, w, "x.", m, 1e9)      # eps so large that the norm is o / sqrt(eps)
    k0, v0 = 2.0 * 0.75, 2.0 * 0.5
    k1, v1 = 4.0 - 0.25 * 2.0, 4.0 - 0.5 * 2.0
    o0, o1 = 3.0 * k0 * v0 * 2.0, (k0 * v0 + 3.0 * k1 * v1) * 4.0
    silu = lambda z: z / (1.0 + math.exp(-z))
    want = [o0 / math.sqrt(1e9 + o0 * o0) * silu(2.0), o1 / math.sqrt(1e9 + o1 * o1) * silu(4.0)]
    assert torch.allclose(out[:, 0], torch.tensor(want).double(), rtol=1e-9)
    # a third token sees the second's decay once on the first product: w of token 1 reads the blend, all of token 0
    out3 = plain.time_mixing(plain.Arithmetic(torch.float64), torch.tensor([[2.0], [4.0], [0.5]]).double(), w, "x.", m, 1e9)
    decay = math.exp(-math.exp(math.tanh(2.0) - 1.0))
    k2, v2 = 0.5 + 0.25 * 3.5, 0.5 + 0.5 * 3.5
    o2 = (decay * k0 * v0 + k1 * v1 + 3.0 * k2 * v2) * 0.5
    assert abs(out3[2, 0].item() - o2 / math.sqrt(1e9 + o2 * o2) * silu(0.5)) < 1e-9


def test_state_space_by_hand():
    """One head of one entry over a state of one: step size, decay, skip, taps oldest first with zeros
    before the start, and the gate ahead of the norm."""
    m = {"heads": 1, "vdim": 1, "state": 1, "groups": 1, "conv": 2, "norm_groups": 1}
    w = {"x.in": torch.tensor([[0.0], [1.0], [1.0], [1.0], [0.0]]).double(),
         "x.conv": torch.tensor([[10.0, 1.0], [0.0, 1.0], [0.0, 1.0]]).double(), "x.conv.b": torch.tensor([0.0, 0.5, 0.0]).double(),
         "x.dt_bias": torch.tensor([0.3]).double(), "x.A_log": torch.tensor([math.log(2.0)]).double(),
         "x.D": torch.tensor([5.0]).double(), "x.norm": torch.ones(1).double(), "x.o": torch.ones(1, 1).double()}
    w["x.in"][0] = 7.0                            # z = 7 h
    h = torch.tensor([[1.0], [2.0]]).double()
    out = plain.state_space(plain.Arithmetic(torch.float64), h, w, "x.", m, 1e9)
    silu = lambda z: z / (1.0 + math.exp(-z))
    x = [silu(1.0), silu(12.0)]
    B, C = [silu(1.5), silu(2.5)], [silu(1.0), silu(2.0)]
    t = math.log1p(math.exp(0.3))
    a = math.exp(-2.0 * t)
    s0 = t * B[0] * x[0]
    s1 = a * s0 + t * B[1] * x[1]
    y = [(s0 * C[0] + 5.0 * x[0]) * silu(7.0), (s1 * C[1] + 5.0 * x[1]) * silu(14.0)]
    want = [v / math.sqrt(v * v + 1e9) for v in y]
    assert torch.allclose(out[:, 0], torch.tensor(want).double(), rtol=1e-9)


def test_latent_attention_of_a_single_token_is_its_value_times_its_gate():
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "kv_rank": 5, "scale": 0.7, "rot": {"base": 10.0, "dims": 2}}
    g = torch.Generator().manual_seed(3)
    w = {"x." + k: torch.randn(*s, generator=g).double() for k, s in
         {"q": (10, 6), "dkv": (7, 6), "dkv.norm": (5,), "uk": (6, 5), "uv": (8, 5), "g": (2, 6), "o": (6, 8)}.items()}
    h = torch.randn(1, 6, generator=g).double()
    out = plain.latent_attention(plain.Arithmetic(torch.float64), h, w, "x.", m, 1e-6, torch.arange(1))
    c = plain.rms_divide((h @ w["x.dkv"].t())[:, :5], 1e-6) * w["x.dkv.norm"]
    v = (c @ w["x.uv"].t()).reshape(2, 4) * plain.logistic(h @ w["x.g"].t()).reshape(2, 1)
    assert torch.allclose(out, v.reshape(1, 8) @ w["x.o"].t(), atol=1e-10)


def test_routing_is_a_softmax_over_the_chosen_and_the_dense_form_squares():
    ar = plain.Arithmetic(torch.float64)
    g = torch.Generator().manual_seed(5)
    w = {"m.router": torch.randn(4, 6, generator=g).double(), "m.up": torch.randn(5, 6, generator=g).double(),
         "m.down": torch.randn(6, 5, generator=g).double()}
    for e in range(4):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"] = torch.randn(3, 6, generator=g).double(), torch.randn(3, 6, generator=g).double()
        w[f"m.e{e}.down"] = torch.randn(6, 3, generator=g).double()
    h = torch.randn(2, 6, generator=g).double()
    chosen, weight, z = plain.route(ar, h, w, "m.", 2)
    a, b = sorted(z[0].tolist(), reverse=True)[:2]
    assert abs(weight[0, 0].item() - 1.0 / (1.0 + math.exp(b - a))) < 1e-12 and abs(weight[0].sum().item() - 1.0) < 1e-12
    out = plain.mixture(ar, h, w, "m.", {"router": {"experts": 4, "top": 2}, "expert": {"ff": 3}})
    assert torch.allclose(out[0], sum(c * plain.expert(ar, h[:1], w, f"m.e{e}.")[0] for e, c in zip(chosen[0].tolist(), weight[0])))
    up = h @ w["m.up"].t()
    assert torch.allclose(plain.dense(ar, h, w, "m."), (torch.relu(up) ** 2) @ w["m.down"].t())
    assert torch.allclose(plain.dense(ar, 2.0 * h, w, "m."), 4.0 * plain.dense(ar, h, w, "m."))
