"""Vozirax on the CPU: configuration, model spec, tensor names, cache and state needs, a folder written and read back,
and properties of the plain mechanisms."""

import copy
import json
import math

import pytest
import torch

import plain_vozirax as plain
from pagedserve_b200.config.registry import ConfigError, resolve_architecture
from pagedserve_b200.config.vozirax import VoziraxConfig, named_config
from pagedserve_b200.models.model import Model, init_plan
from pagedserve_b200.models.vozirax import build_vozirax_spec
from pagedserve_b200.parts.base import PartEnv

M, D, X, E = plain.mamba_layer, plain.diff_layer, plain.dense_mlp, plain.moe_mlp
CONFIG = plain.make_config(
    [M(6, 16, 24, groups=3, norm_groups=2, conv=3, mlp=E(6, 2, 20)), D(4, 2, 12, 20, mlp=X(40)),
     D(8, 2, 12, 20, q_temp=None, kv_from=1, mlp=E(4, 3, 24, groups=None)), M(2, 20, 10, groups=1, norm_groups=1, conv=1),
     D(3, 3, 10, 44, diff=-0.2)], width=56, vocab=89)


def cpu_model(values, dtype=torch.float32):
    spec = build_vozirax_spec(VoziraxConfig.from_dict(values))
    return spec, Model(spec, PartEnv(ops=None, dtype=dtype, device="cpu"))


def test_config_round_trip_and_registry():
    name, config_class, builder = resolve_architecture(CONFIG)
    assert name == "Vozirax" and config_class is VoziraxConfig and builder is build_vozirax_spec
    config = VoziraxConfig.from_dict(CONFIG)
    assert config.to_dict() == CONFIG
    assert VoziraxConfig.from_dict(config.to_dict()).to_dict() == CONFIG
    assert config.vocabulary_size == 89 and config.logit_scale == 0.7 and config.max_model_len >= 1 << 24


def test_keys_that_may_be_absent():
    values = copy.deepcopy(CONFIG)
    values["layers"][4]["mixer"].pop("kv_heads")
    values["layers"][4]["mixer"].pop("vdim")
    values["layers"][2]["mlp"]["router"].pop("scale")
    values["layers"][3].pop("mlp")
    config = VoziraxConfig.from_dict(values)
    assert config.layers[4]["mixer"]["kv_heads"] == 3 and config.layers[4]["mixer"]["vdim"] == 10
    assert config.layers[2]["mlp"]["router"]["scale"] == 1.0 and config.layers[3]["mlp"] is None


@pytest.mark.parametrize("change", [
    lambda c: c.update(vocab=0), lambda c: c.update(width=-3), lambda c: c.pop("norm"), lambda c: c["norm"].update(eps=0),
    lambda c: c.pop("logit_scale"), lambda c: c.update(logit_scale="x"), lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0].pop("mixer"),
    lambda c: c["layers"][0]["mixer"].update(groups=4), lambda c: c["layers"][0]["mixer"].update(norm_groups=5),
    lambda c: c["layers"][0]["mixer"].update(conv=0), lambda c: c["layers"][0]["mixer"].update(conv=17),
    lambda c: c["layers"][0]["mixer"].update(state=600), lambda c: c["layers"][0]["mixer"].pop("state"),
    lambda c: c["layers"][1]["mixer"].update(heads=3), lambda c: c["layers"][1]["mixer"].update(dim=600),
    lambda c: c["layers"][1]["mixer"].pop("scale"), lambda c: c["layers"][1]["mixer"].pop("diff"),
    lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), lambda c: c["layers"][1]["mixer"]["q_temp"].pop("coef"),
    lambda c: c["layers"][2]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=0),
    lambda c: c["layers"][2]["mixer"].update(dim=16), lambda c: c["layers"][2]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][4]["mixer"].update(kv_from=2, kv_heads=3),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"), lambda c: c["layers"][1]["mlp"].pop("ff"),
    lambda c: c["layers"][0]["mlp"].pop("expert"), lambda c: c["layers"][0]["mlp"].pop("router"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["layers"][0]["mlp"]["router"].update(experts=7),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), lambda c: c["layers"][2]["mlp"]["router"].update(top=5)])
def test_inconsistent_configurations_are_refused(change):
    values = copy.deepcopy(CONFIG)
    change(values)
    with pytest.raises(ConfigError):
        VoziraxConfig.from_dict(values)


def test_spec_needs_and_tensor_names():
    spec, model = cpu_model(CONFIG, torch.bfloat16)
    needs, states = model.kv_needs(), model.state_needs()
    # two keys of 12 beside values of 20 take 32 numbers in a bfloat16 cache, two of 10 beside values of 44 take 48; the layer
    # that borrows has no cache layer of its own
    assert [None if n is None else (n.n_kv_heads, n.head_dim, n.window, n.planes) for n in needs] == [
        None, (2, 32, None, 2), None, None, (3, 48, None, 2)]
    assert [(entry.layer, entry.cache_layer) for entry in spec.schedule] == [(0, 0), (1, 1), (2, 1), (3, 3), (4, 4)]
    # kept rows of the convolution (two of 96 + 2 * 72 channels), then 6 matrices of 24 x 16; one tap keeps nothing
    assert [None if s is None else s.shape for s in states] == [(2 * 240 + 6 * 24 * 16,), None, None, (2 * 10 * 20,), None]
    assert model.graph_safe
    assert cpu_model(CONFIG)[1].kv_needs()[1].head_dim == 24           # float32 is not rounded up
    names = {spec.checkpoint_name(param.name): tuple(param.shape) for param, _ in init_plan(spec)}
    assert names == {name: tuple(shape) for name, shape in plain.tensor_shapes(CONFIG).items()}
    assert spec.normalise_name("l3.norm2") == "l3.norm2.weight" and spec.normalise_name("l3.mix.norm") == "l3.mix.norm"
    assert spec.normalise_name("head") == "head.weight"


def test_a_model_folder_loads_and_a_wrong_one_is_refused(tmp_path):
    from pagedserve_b200.weights.loader import WeightError
    from pagedserve_b200.weights.safetensors_io import write_safetensors

    tensors = plain.random_model(CONFIG, seed=3)
    spec, model = cpu_model(CONFIG)
    with open(tmp_path / "config.json", "w") as handle:
        json.dump(CONFIG, handle)
    write_safetensors(str(tmp_path / "model.safetensors"), tensors)
    model.load_folder(str(tmp_path))
    # factors reach the parts that apply them, the logits' factor sits in the last norm's gain
    assert torch.equal(model.blocks[0].mixer.result_factor, tensors["l0.ls1"].float())
    assert torch.equal(model.blocks[2].feed_forward.result_factor, tensors["l2.ls2"].float())
    assert torch.allclose(model.final_norm.weight, (1.0 + tensors["final.norm"].float()) * 0.7)
    double = {name: t.double() for name, t in tensors.items()}
    for index in (1, 2, 4):
        want = float(plain.map_share(double, f"l{index}.mix.", CONFIG["layers"][index]["mixer"]))
        assert math.isclose(model.blocks[index].mixer.share, want, rel_tol=1e-9)
    mixer = model.blocks[4].mixer                                       # every part begins on a multiple of eight rows
    assert (mixer.k_offset, mixer.v_offset, mixer.gate_offset) == (64, 128, 264) and mixer.w_in.shape[0] == 272
    read, config = plain.read_folder(str(tmp_path))
    assert config == CONFIG and all(torch.equal(read[name], tensors[name].double()) for name in tensors)
    broken = dict(tensors)
    broken["l0.mix.dt_bias"] = torch.ones(5).to(torch.bfloat16)
    broken["l2.mix.k"] = tensors["l1.mix.k"]                            # a borrowing layer has no keys
    broken.pop("l1.mix.lq2")
    with pytest.raises(WeightError) as error:
        model.load_tensors(broken)
    assert "l1.mix.lq2" in str(error.value) and "l2.mix.k" in str(error.value)
    assert error.value.wrong_shape[0][0] == "l0.mix.dt_bias"


def test_a_random_model_folder_reads_back(tmp_path):
    from pagedserve_b200.weights.random_init import write_random_model

    config = named_config("vozirax-tiny")
    folder = write_random_model(str(tmp_path), config, seed=7)
    tensors, read_config = plain.read_folder(folder)
    logits = plain.forward(tensors, read_config, [3, 1, 4, 1, 5, 9, 2, 6])
    assert logits.shape == (8, config.vocab) and torch.isfinite(logits).all()
    _, model = cpu_model(read_config)
    model.load_folder(folder)                                   # every tensor found, shaped and cast


def test_parts_that_cannot_apply_a_factor_refuse_it():
    from pagedserve_b200.models.spec import PartSpec
    from pagedserve_b200.parts import create_part

    env = PartEnv(ops=None, dtype=torch.float32, device="cpu")
    with_bias = create_part("feed_forward", PartSpec("dense_mlp", dict(
        hidden_size=8, inner_size=8, activation="gelu_tanh", up_name="up", down_name="down")), env)
    with pytest.raises(ValueError):
        with_bias.set_result_factor(torch.ones(8))
    with pytest.raises(ValueError):                              # a norm with a mean
        norm = create_part("norm", PartSpec("layernorm", dict(width=8, eps=1e-5, name="n")), env)
        create_part("block", PartSpec("parallel_pre_norm", dict(scales={})), env, mixer=cpu_model(CONFIG)[1].blocks[0].mixer,
                    feed_forward=with_bias,
                    norms={"pre_mixer": norm, "pre_feed_forward": norm})
    with pytest.raises(ValueError):                              # experts without a gate have no shared expert
        create_part("feed_forward", PartSpec("routed_experts", dict(
            hidden_size=8, n_experts=4, expert_ff=8, top=1, shared_ff=8, expert_form=dict(kind="relu_squared"))), env)


@pytest.mark.parametrize("width", [64, 37, 2])
def test_position_frequencies_match_the_part(width):
    from pagedserve_b200.parts.positions import SinusoidalPositions

    part = SinusoidalPositions(dict(hidden_size=width, base=10000.0), "", PartEnv(ops=None, dtype=torch.float32, device="cpu"))
    table = part.sinusoids().double()
    exact = torch.tensor([10000.0 ** (-2.0 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64)
    assert torch.allclose(table[:, 0] + table[:, 1], exact, rtol=1e-12, atol=0)
    rows = plain.position_rows(torch.tensor([0, 1, 5000]), width)
    assert torch.allclose(rows[0, 0::2], torch.zeros(len(rows[0, 0::2])).double()) and bool((rows[0, 1::2] == 1.0).all())
    angle = 5000.0 * exact
    assert torch.allclose(rows[2, 0::2], torch.sin(angle)) and torch.allclose(rows[2, 1::2], torch.cos(angle)[:width // 2])


def test_properties_of_the_plain_mechanisms():
    g = torch.Generator().manual_seed(0)
    randn = lambda *shape: torch.randn(*shape, generator=g, dtype=torch.float64)
    # a convolution with the last tap alone scales each row, its first tap of three reaches two tokens back
    u = randn(6, 2)
    assert torch.equal(plain.causal_convolution(u, torch.tensor([[0.0, 0.0, 2.0]] * 2).double(), torch.zeros(2).double()), 2.0 * u)
    shifted = plain.causal_convolution(u, torch.tensor([[1.0, 0.0, 0.0]] * 2).double(), torch.ones(2).double()) - 1.0
    assert torch.allclose(shifted[2:], u[:-2]) and float(shifted[:2].abs().max()) == 0.0
    # the state as the sum that the recurrence stands for
    T, H, G, N, e = 7, 4, 2, 3, 5
    x, b, c, dt = randn(T, H, e), randn(T, G, N), randn(T, G, N), torch.rand(T, H, generator=g).double() + 0.1
    a_log, d = randn(H), randn(H)
    got = plain.state_space(x, b, c, dt, a_log, d)
    for h in range(H):
        for t in range(T):
            want = d[h] * x[t, h]
            for s in range(t + 1):
                decay = torch.exp(-torch.exp(a_log[h]) * dt[s + 1:t + 1, h].sum())
                want = want + decay * dt[s, h] * (b[s, h // 2] @ c[t, h // 2]) * x[s, h]
            assert torch.allclose(got[t, h], want)
    assert torch.allclose(plain.softplus(torch.tensor([-900.0, 0.0, 900.0]).double()), torch.tensor([0.0, math.log(2.0), 900.0]).double())
    # parts of a row are normed by themselves
    row = torch.cat([randn(4), 1000.0 * randn(4)])[None]
    parts = plain.unit_rms_in_parts(row, 2, 1e-12)
    assert torch.allclose((parts.reshape(2, 4) ** 2).mean(-1), torch.ones(2).double())
    # the temperature rises at multiples of `every`, counted from one
    warm = plain.temperature(torch.arange(9), {"coef": 0.5, "every": 4})
    assert torch.allclose(warm, 1.0 + 0.5 * torch.log(torch.tensor([1, 1, 1, 2, 2, 2, 2, 3, 3]).double()))
    # equal maps leave (1 - share) of one of them, whose norm does not know the factor
    config = plain.make_config([D(2, 1, 6, 10, q_temp=None)], width=24)
    tensors = {name: t.double() for name, t in plain.random_model(config, seed=2).items()}
    m, rows, eps = config["layers"][0]["mixer"], randn(5, 24), 1e-12
    for name in ("q", "k"):
        w = tensors["l0.mix." + name].reshape(-1, 2, 6, 24)
        w[:, 1] = w[:, 0]
    tensors["l0.mix.o"] = torch.eye(20, dtype=torch.float64)[:, :20]
    kv = plain.keys_and_values(tensors, "l0.mix.", m, rows, eps)
    got = plain.differential_attention(tensors, "l0.mix.", m, rows, torch.arange(5), eps, kv)
    gates = torch.sigmoid(rows @ tensors["l0.mix.g"].T)
    sign = torch.sign(1.0 - plain.map_share(tensors, "l0.mix.", m))
    first = sign * plain.unit_rms(kv[1][0, 0], eps) * (1.0 - m["diff"])     # the first token sees its own value alone
    assert torch.allclose(got[0].reshape(2, 10), first[None] * gates[0][:, None])
    # a closed group is out even where the standing experts' choice scores are negative
    scores = torch.tensor([0.9, 0.1, 0.2, 0.3], dtype=torch.float64)
    correction = torch.tensor([-2.0, -2.0, -0.9, -0.9], dtype=torch.float64)
    weights, margin = plain.election(scores, correction, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}, "scale": 3.0})
    assert set(weights) == {2, 3} and math.isclose(float(sum(weights.values())), 3.0) and margin > 0
    assert math.isclose(float(weights[3] / weights[2]), 1.5)
    # a group is marked by its two largest, not by its largest
    scores = torch.tensor([0.9, 0.1, 0.6, 0.6], dtype=torch.float64)
    weights, _ = plain.election(scores, torch.zeros(4).double(), {"experts": 4, "top": 1, "groups": {"count": 2, "keep": 1}})
    assert set(weights) == {2}
