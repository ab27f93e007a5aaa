"""Suvunex on the CPU: configuration, model spec, tensor names, cache and state needs, a folder written and read back,
and properties of the plain mechanisms."""

import copy
import math

import pytest
import torch

import plain_suvunex as plain
from pagedserve_b200.config.registry import ConfigError, resolve_architecture
from pagedserve_b200.config.suvunex import SuvunexConfig, named_config
from pagedserve_b200.models.model import Model, init_plan
from pagedserve_b200.models.suvunex import build_suvunex_spec
from pagedserve_b200.parts.base import PartEnv

P, L, R, T, X = plain.parallel_layer, plain.left_side, plain.right_side, plain.talking_layer, plain.dense_mlp
CONFIG = plain.make_config(
    [P(L(4, 2, 16, 24, rot_dims=8, scaling=plain.llama_scaling(4.0, 1.0, 4.0, 64)), R(3, 16, 24, tau=8.0), mlp=X(48)),
     T(6, 3, 16, rot_dims=10, factor=4.0, mlp=X(40)),
     P(L(3, 3, 20, 12, rot_dims=0), R(5, 10, 14, tau=0.5), left_scale=-0.4, right_scale=1.5, mlp=None),
     T(3, 1, 20, mlp=None)],
    width=64, vocab=97, taps=3)


def cpu_model(values, dtype=torch.float32):
    spec = build_suvunex_spec(SuvunexConfig.from_dict(values))
    return spec, Model(spec, PartEnv(ops=None, dtype=dtype, device="cpu"))


def test_config_round_trip_and_registry():
    name, config_class, builder = resolve_architecture(CONFIG)
    assert name == "Suvunex" and config_class is SuvunexConfig and builder is build_suvunex_spec
    config = SuvunexConfig.from_dict(CONFIG)
    assert config.to_dict() == CONFIG
    assert SuvunexConfig.from_dict(config.to_dict()).to_dict() == CONFIG
    assert config.vocabulary_size == 97 and config.canon_taps == 3 and config.logit_scale == 0.5


def test_keys_that_may_be_absent():
    values = copy.deepcopy(CONFIG)
    values["layers"][1]["mixer"].pop("vdim")
    values["layers"][2]["mixer"]["left"].pop("kv_heads")
    values["layers"][3]["mixer"].pop("rot")
    config = SuvunexConfig.from_dict(values)
    assert config.layers[1]["mixer"]["vdim"] == 16 and config.layers[2]["mixer"]["left"]["kv_heads"] == 3
    assert config.layers[3]["mixer"]["rot"] is None and "rot" not in config.to_dict()["layers"][3]["mixer"]


@pytest.mark.parametrize("change", [
    lambda c: c.update(vocab=0), lambda c: c.update(width=-3), lambda c: c.pop("norm"), lambda c: c["norm"].update(eps=0),
    lambda c: c.pop("canon"), lambda c: c["canon"].update(taps=0), lambda c: c["canon"].update(taps=17),
    lambda c: c.pop("embedding"), lambda c: c.pop("logit_scale"), lambda c: c.update(logit_scale="x"),
    lambda c: c.update(layers=[]), lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0].pop("mixer"),
    lambda c: c["layers"][0]["mixer"].pop("left"), lambda c: c["layers"][0]["mixer"]["left"].update(heads=3),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=300), lambda c: c["layers"][0]["mixer"]["left"].pop("scale"),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("low"),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(low=4.0),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(fast=1.0),
    lambda c: c["layers"][0]["mixer"].pop("right"), lambda c: c["layers"][0]["mixer"]["right"].update(tau=0),
    lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"), lambda c: c["layers"][0]["mixer"].pop("right_scale"),
    lambda c: c["layers"][1]["mixer"].update(vdim=8), lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=-1),
    lambda c: c["layers"][1]["mlp"].update(kind="moe"), lambda c: c["layers"][1]["mlp"].pop("ff")])
def test_inconsistent_configurations_are_refused(change):
    values = copy.deepcopy(CONFIG)
    change(values)
    with pytest.raises(ConfigError):
        SuvunexConfig.from_dict(values)


def test_spec_needs_and_tensor_names():
    spec, model = cpu_model(CONFIG, torch.bfloat16)
    needs, states = model.kv_needs(), model.state_needs()
    # heads of 16 keys and 24 values take 32 numbers in a bfloat16 cache, keys that are values 16 (10 -> 16) as well
    assert [(n.n_kv_heads, n.head_dim, n.window, n.chunk, n.planes) for n in needs] == [
        (2, 32, None, None, 2), (3, 16, None, None, 2), (3, 32, None, None, 2), (1, 32, None, None, 2)]
    # the kept rows of the convolution in every layer, then the recurrence's matrices
    assert [s.shape for s in states] == [(2 * 64 + 3 * 16 * 24,), (2 * 64,), (2 * 64 + 5 * 10 * 14,), (2 * 64,)]
    assert model.graph_safe
    names = {spec.checkpoint_name(param.name): tuple(drawn[2] if len(drawn) > 2 else param.shape)
             for param, drawn in init_plan(spec)}
    want = {name: tuple(shape) for name, shape in plain.tensor_shapes(CONFIG).items()}
    for index in (0, 2):                                        # the decay's inner size is what a file has
        want[f"l{index}.mix.right.a1"] = (16, 64)
        want[f"l{index}.mix.right.a2"] = (want[f"l{index}.mix.right.a2"][0], 16)
    assert names == want
    assert spec.normalise_name("l3.norm1b") == "l3.norm1b.weight" and spec.normalise_name("l3.mix.q.norm") == "l3.mix.q.norm"
    assert spec.normalise_name("head") == "head.weight"


def test_one_tap_keeps_nothing():
    values = copy.deepcopy(CONFIG)
    values["canon"]["taps"] = 1
    _, model = cpu_model(values)
    states = model.state_needs()
    assert states[1] is None and states[0].shape == (3 * 16 * 24,)


def test_a_model_folder_loads_and_a_wrong_one_is_refused(tmp_path):
    import json

    from pagedserve_b200.weights.loader import WeightError
    from pagedserve_b200.weights.safetensors_io import write_safetensors

    tensors = plain.random_model(CONFIG, seed=3)
    spec, model = cpu_model(CONFIG)
    with open(tmp_path / "config.json", "w") as handle:
        json.dump(CONFIG, handle)
    write_safetensors(str(tmp_path / "model.safetensors"), tensors)
    model.load_folder(str(tmp_path))
    mixer = model.blocks[2].mixer
    # scales are not rounded into matrices: the attention's is left to the block, the recurrence's is relative to it
    assert mixer.output_scale == -0.4 and mixer.scales == [-0.4, 1.5]
    heads = mixer.w_out[:, :60].reshape(64, 3, 20)              # heads of 20 keys and 12 values: padded to 20
    assert torch.equal(heads[:, :, :12].reshape(64, 36), tensors["l2.mix.left.o"].float())
    assert float(heads[:, :, 12:].abs().max()) == 0.0
    assert torch.allclose(mixer.b_out, tensors["l2.mix.left.o.b"].float())
    read, config = plain.read_folder(str(tmp_path))
    assert config == CONFIG and all(torch.equal(read[name], tensors[name].double()) for name in tensors)
    broken = dict(tensors)
    broken["l0.norm1"] = torch.ones(64).to(torch.bfloat16)      # a gain per coordinate where one number is wanted
    broken.pop("l1.mix.talk")
    with pytest.raises(WeightError) as error:
        model.load_tensors(broken)
    assert "l1.mix.talk" in str(error.value) and error.value.wrong_shape[0][0] == "l0.norm1"


def test_a_random_model_folder_reads_back(tmp_path):
    from pagedserve_b200.weights.random_init import write_random_model

    config = named_config("suvunex-tiny")
    folder = write_random_model(str(tmp_path), config, seed=7)
    tensors, read_config = plain.read_folder(folder)
    logits = plain.forward(tensors, read_config, [3, 1, 4, 1, 5, 9, 2, 6])
    assert logits.shape == (8, config.vocab) and torch.isfinite(logits).all()
    _, model = cpu_model(read_config)
    model.load_folder(folder)                                   # every tensor found, shaped and cast


def test_a_scale_of_zero_takes_a_mixer_out():
    values = copy.deepcopy(CONFIG)
    values["layers"][0]["mixer"]["left_scale"] = 0.0
    _, model = cpu_model(values)
    model.load_tensors(plain.random_model(values, seed=1))
    mixer = model.blocks[0].mixer
    assert mixer.output_scale == 1.0 and float(mixer.w_out[:, :4 * 24].abs().max()) == 0.0
    assert float(mixer.b_out.abs().max()) == 0.0


def test_blocks_that_do_not_scale_refuse_such_a_mixer():
    from pagedserve_b200.models.spec import PartSpec
    from pagedserve_b200.parts import create_part

    env = PartEnv(ops=None, dtype=torch.float32, device="cpu")
    spec, model = cpu_model(CONFIG)
    with pytest.raises(ValueError):
        create_part("block", PartSpec("pre_norm"), env, mixer=model.blocks[0].mixer,
                    feed_forward=model.blocks[0].feed_forward, norms={})
    create_part("block", PartSpec("pre_norm"), env, mixer=model.blocks[1].mixer, feed_forward=model.blocks[1].feed_forward,
                norms={})


def test_frequencies_match_the_part():
    from pagedserve_b200.parts.positions import RotaryPositions

    for dims, base, scaling in ((16, 10000.0, plain.llama_scaling(4.0, 1.0, 4.0, 64)), (6, 100.0, None), (24, 500.0, {"factor": 3.0}),
                                (64, 500000.0, plain.llama_scaling(8.0, 1.0, 4.0, 8192)), (40, 30.0, plain.llama_scaling(2.0, 0.5, 9.0, 100)),
                                (0, 10000.0, {"factor": 2.0})):
        part = RotaryPositions(dict(dims=dims, base=base, interleaved=False, head_dim=max(dims, 8), scaling=scaling), "",
                               PartEnv(ops=None, dtype=torch.float32, device="cpu"))
        want = plain.pair_frequencies({"dims": dims, "base": base, "scaling": scaling})
        split = part.inv_freq_split().double()
        assert torch.allclose(split[:, 0] + split[:, 1], want, rtol=1e-12, atol=0)
        assert part.amplitude == 1.0
    # fast pairs stay, slow ones are divided, and some lie between
    scaled = plain.pair_frequencies({"dims": 64, "base": 10000.0, "scaling": plain.llama_scaling(8.0, 1.0, 4.0, 512)})
    bare = plain.pair_frequencies({"dims": 64, "base": 10000.0})
    ratio = scaled / bare
    assert torch.allclose(ratio[:3], torch.ones(3).double()) and torch.allclose(ratio[-8:], torch.full((8,), 0.125).double())
    assert ((ratio > 0.13) & (ratio < 0.99)).any() and (ratio[1:] <= ratio[:-1] + 1e-12).all()
    with pytest.raises(ValueError):
        RotaryPositions(dict(dims=8, base=10.0, head_dim=8, scaling={"factor": 2.0, "low": 1.0}), "",
                        PartEnv(ops=None, dtype=torch.float32, device="cpu"))


def test_properties_of_the_plain_mechanisms():
    g = torch.Generator().manual_seed(0)
    # a convolution whose last tap alone is one doubles what it reads; the first tap of three reaches two tokens back
    h = torch.randn(6, 2, generator=g, dtype=torch.float64)
    assert torch.equal(plain.with_convolution(h, torch.tensor([[0.0, 0.0, 1.0]] * 2, dtype=torch.float64)), 2.0 * h)
    shifted = plain.with_convolution(h, torch.tensor([[1.0, 0.0, 0.0]] * 2, dtype=torch.float64)) - h
    assert torch.allclose(shifted[2:], h[:-2]) and float(shifted[:2].abs().max()) == 0.0
    # a one in the denominator: a single key of score s has weight e^s / (1 + e^s)
    weights = plain.causal_softmax(torch.tensor([[[0.3]]], dtype=torch.float64), torch.zeros(1))
    assert math.isclose(float(weights), math.exp(0.3) / (1.0 + math.exp(0.3)), rel_tol=1e-12)
    # turning keeps a head's length, so dividing by it commutes with turning
    x = torch.randn(5, 3, 16, generator=g, dtype=torch.float64)
    rot, positions = {"dims": 10, "base": 100.0}, torch.arange(5)
    assert torch.allclose(plain.unit_rms(plain.rotate_halves(x, positions, rot), 1e-5),
                          plain.rotate_halves(plain.unit_rms(x, 1e-5), positions, rot))
    # mixing the weights by the identity leaves plain attention; by a permutation of heads of one group it swaps weights
    config = plain.make_config([T(4, 1, 8)], width=24)
    tensors = {name: t.double() for name, t in plain.random_model(config, seed=2).items()}
    rows = torch.randn(7, 24, generator=g, dtype=torch.float64)
    tensors["l0.mix.o"] = torch.eye(32, dtype=torch.float64)[:24]
    tensors["l0.mix.talk"] = torch.eye(4, dtype=torch.float64)
    own = plain.talking_attention(tensors, "l0.mix.", config["layers"][0]["mixer"], rows, torch.arange(7), 1e-5)
    tensors["l0.mix.talk"] = torch.eye(4, dtype=torch.float64)[[1, 0, 2, 3]]
    swapped = plain.talking_attention(tensors, "l0.mix.", config["layers"][0]["mixer"], rows, torch.arange(7), 1e-5)
    assert torch.allclose(swapped[:, :8], own[:, 8:16]) and torch.allclose(swapped[:, 16:], own[:, 16:])
    # the recurrence with decays near one is a running sum of k v^T
    m = {"heads": 1, "dim": 4, "vdim": 3, "tau": 1e9}
    tensors = {"q": torch.eye(4).double(), "k": torch.eye(4).double(), "v": torch.randn(3, 4, generator=g).double(),
               "g": torch.randn(3, 4, generator=g).double(), "o": torch.eye(3).double(), "norm": torch.ones(3).double(),
               "a1": torch.ones(1, 4).double(), "a2": torch.ones(4, 1).double(), "a2.b": torch.zeros(4).double()}
    rows = torch.randn(5, 4, generator=g, dtype=torch.float64)
    got = plain.gated_linear_attention(tensors, "", m, rows, 1e-12)
    v = rows @ tensors["v"].T
    summed = torch.stack([sum((rows[t] @ rows[s]) * v[s] for s in range(t + 1)) for t in range(5)]) * 0.5
    gate = rows @ tensors["g"].T
    assert torch.allclose(got, plain.unit_rms(summed, 1e-12) * gate * torch.sigmoid(gate), atol=1e-6)
