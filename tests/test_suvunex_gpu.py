"""Suvunex in the engine against the plain implementation (tests/plain_suvunex.py): every mechanism alone, then whole
models through the step function, the trace replay and the scheduler, in float32 and bfloat16.

The configurations are made here, with random weights; sizes differ from model to model so that nothing rests on a
value that happens to be 1 or on two sizes that happen to be equal."""

import io
import json
import os
import tempfile
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import helpers
import plain_suvunex as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"

P, L, R, T, X = plain.parallel_layer, plain.left_side, plain.right_side, plain.talking_layer, plain.dense_mlp
slow = plain.llama_scaling
# both mixers, two and three key heads, values larger than keys (a cached head is padded), different sizes on the two
# sides, layers without a feed-forward
CONFIG_A = plain.make_config(
    [P(L(4, 2, 16, 24, rot_dims=8, scaling=slow(4.0, 1.0, 4.0, 64)), R(3, 16, 24, tau=8.0), mlp=X(48)),
     T(6, 3, 16, rot_dims=10, factor=4.0, mlp=X(40)),
     P(L(4, 1, 16, 16, base=500.0), R(2, 24, 16, tau=1.0), left_scale=1.2, right_scale=0.3, mlp=None),
     T(4, 2, 32, base=100.0, scale=0.2, mlp=X(72)),
     T(5, 5, 16, factor=2.0, scale=0.3, mlp=None)],
    width=64, vocab=97, taps=3)
# heads of 64 and 128 numbers (the tensor-core attention kernels), mixed heads among them, four taps
CONFIG_B = plain.make_config(
    [T(4, 2, 64, rot_dims=32, base=500.0, factor=8.0, scale=0.11, mlp=X(160)),
     P(L(6, 3, 64, 64, rot_dims=48, base=250000.0, scaling=slow(8.0, 1.0, 4.0, 256), scale=0.5), R(4, 64, 64), mlp=X(96)),
     P(L(2, 2, 128, 128, scale=0.3), R(1, 128, 128, tau=4.0), left_scale=0.4, right_scale=0.9, mlp=None),
     T(2, 1, 128, base=250000.0, scale=0.07, mlp=X(128))],
    width=128, vocab=211, eps=1e-6, taps=4, embedding_scale=9.0, logit_scale=0.3)
# nothing a multiple of 8 or 16, no turning, as many key heads as query heads, single heads, fast decays
CONFIG_C = plain.make_config(
    [P(L(3, 3, 20, 12, rot_dims=6, scale=0.6), R(5, 10, 14, tau=0.5), mlp=X(36)),
     T(3, 1, 10, rot_dims=6, scale=0.3, mlp=None),
     P(L(6, 2, 10, 24, rot_dims=0, scale=0.3), R(1, 36, 20, tau=30.0), mlp=X(50)),
     T(6, 2, 20, rot_dims=0, scale=0.2, mlp=X(20)),
     T(1, 1, 44, base=100.0, factor=3.0, scale=0.15, mlp=None)],
    width=72, vocab=53, eps=1e-4, taps=2)
# one tap (a factor per channel, nothing kept), scales that are negative and zero, eight key heads whose weights are mixed
CONFIG_D = plain.make_config(
    [P(L(5, 1, 80, 48, rot_dims=20, scale=0.2), R(3, 48, 80, tau=2.0), left_scale=-0.6, right_scale=0.8, mlp=X(120)),
     T(8, 8, 16, factor=1.0, scale=0.3, mlp=X(64)),
     P(L(2, 2, 32, 32), R(2, 40, 32), left_scale=0.0, right_scale=-0.5, mlp=X(32)),
     P(L(4, 4, 32, 16), R(2, 8, 8), left_scale=0.8, right_scale=0.0, mlp=None)],
    width=96, vocab=131, eps=1e-3, taps=1, logit_scale=1.7)
# one layer of each kind alone; heads of the recurrence too large for the kernel that keeps them in registers
CONFIG_E = plain.make_config([P(L(2, 1, 16, 16), R(4, 20, 36), mlp=X(24))], width=48, vocab=61, taps=5)
CONFIG_F = plain.make_config([T(3, 3, 24, rot_dims=4, mlp=X(8))], width=40, vocab=77, taps=3)
CONFIG_W = plain.make_config([P(L(2, 1, 16, 16), R(2, 144, 160, tau=4.0), mlp=None),
                              P(L(2, 1, 16, 16), R(1, 32, 136, tau=4.0), mlp=None)], width=56, vocab=41, taps=3)
# layers for keys that stand out: steep scores, and nothing but attention in the first layer's result
CONFIG_S = plain.make_config(
    [P(L(4, 2, 16, 16, rot_dims=8, scale=0.8, scaling=slow(4.0, 1.0, 4.0, 128)), R(1, 8, 8), left_scale=1.0, right_scale=0.0),
     P(L(4, 2, 64, 64, rot_dims=32, base=500.0, scale=0.25), R(1, 8, 8), left_scale=1.0, right_scale=0.0),
     T(4, 2, 32, rot_dims=16, factor=2.0, scale=0.18),
     T(4, 2, 64, factor=4.0, scale=0.12),
     T(6, 3, 20, scale=0.25)],
    width=96, vocab=67, taps=3)
# layers as wide as a small model's (the tensor-core products and prompt attention run at these sizes)
CONFIG_M = plain.make_config(
    [P(L(10, 2, 64, 64, rot_dims=40, scaling=slow(8.0, 1.0, 4.0, 512), scale=0.4), R(5, 64, 96, tau=12.0), mlp=X(700)),
     T(8, 4, 64, factor=8.0, scale=0.125, mlp=X(640)),
     P(L(8, 4, 80, 80, scale=0.3), R(8, 40, 64, tau=16.0), mlp=X(500)),
     T(12, 2, 48, rot_dims=32, base=250000.0, scale=0.15, mlp=None)],
    width=512, vocab=700, eps=1e-6, taps=4)

CONFIGS = {"a": (CONFIG_A, 1, 16), "b": (CONFIG_B, 2, 16), "c": (CONFIG_C, 3, 8), "d": (CONFIG_D, 4, 32),   # config, seed, page
           "e": (CONFIG_E, 5, 16), "f": (CONFIG_F, 6, 8), "w": (CONFIG_W, 7, 16), "s": (CONFIG_S, 8, 16),
           "m": (CONFIG_M, 9, 16)}

_FOLDERS, _TENSORS, _LOGITS = {}, {}, {}


def folder_of(which):
    if which not in _FOLDERS:
        from pagedserve_b200.weights.safetensors_io import write_safetensors

        config, seed, _ = CONFIGS[which]
        holder = tempfile.TemporaryDirectory(prefix=f"ps_suvunex_{which}_")
        tensors = plain.random_model(config, seed)
        if which == "s":                                             # large query gains: one key can stand out
            for name in tensors:
                if name.endswith("mix.q.norm"):
                    tensors[name] = (tensors[name].float() * 3.0).to(torch.bfloat16)
        _TENSORS[which] = tensors
        with open(os.path.join(holder.name, "config.json"), "w") as handle:
            json.dump(config, handle)
        write_safetensors(os.path.join(holder.name, "model.safetensors"), tensors)
        _FOLDERS[which] = holder
    return _FOLDERS[which].name


def plain_logits(which, sequences):
    folder_of(which)
    out = {}
    for name, tokens in sequences.items():
        key = (which, tuple(tokens))
        if key not in _LOGITS:
            _LOGITS[key] = plain.forward(_TENSORS[which], CONFIGS[which][0], tokens).numpy()
        out[name] = _LOGITS[key]
    return out


def assert_rows_close(got, want, dtype, what):
    """float32: every logit within 3e-5 of the scale (sums differ in order only), the best token the same.
    bfloat16: a row's error is the root mean square over the vocabulary against that of the logits; rounding alone
    gives about 1 % in the mean over the rows and a few per cent at single rows, while a wrong key, a lost state or a
    sink left out moves a row by 30 % and more."""
    assert got.shape == want.shape and np.isfinite(got).all(), what
    if dtype == "float32":
        scale = float(np.abs(want).max())
        error = np.abs(got.astype(np.float64) - want).max(-1)
        assert float(error.max()) <= 3e-5 * scale, \
            f"{what}: row {int(error.argmax())} is off by {float(error.max()):.3e}, scale {scale:.3e}"
        ordered = np.sort(want, axis=-1)
        clear = (ordered[:, -1] - ordered[:, -2]) > 1e-4 * scale
        assert (got.argmax(-1) == want.argmax(-1))[clear].all(), f"{what}: another best token"
        return
    error = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
    assert float(error.max()) < 0.12, f"{what}: row {int(error.argmax())} is off by {float(error.max()):.3f}"
    assert float(error.mean()) < 0.025, f"{what}: rows are off by {float(error.mean()):.4f} in the mean"


def build_engine(which, dtype, **options):
    from pagedserve_b200.config.engine_config import EngineConfig
    from pagedserve_b200.engine.engine import Engine

    defaults = dict(dtype=dtype, block_size=CONFIGS[which][2], num_blocks=96, max_num_seqs=4, max_model_len=512)
    defaults.update(options)
    return Engine.from_folder(folder_of(which), EngineConfig(**defaults))


def sequences_for(which, lengths, seed=0):
    vocab = CONFIGS[which][0]["vocab"]
    return {f"s{i}": helpers.random_tokens(vocab, n, seed=seed + i) for i, n in enumerate(lengths)}


def rel_err(got, want):
    want = want.double()
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-30))


# ------------------------------------------------------------------ the replay program on whole models
def run_replay(which, dtype, steps, slots=4):
    from pagedserve_b200.engine import replay as replay_module

    with tempfile.TemporaryDirectory(prefix="ps_out_") as out:
        args = SimpleNamespace(model=folder_of(which), dtype=dtype, out=out, max_tokens=helpers.peak_tokens(steps),
                               block_size=CONFIGS[which][2], max_num_seqs=slots, disable_cuda_graphs=False)
        stdin = io.StringIO("".join(json.dumps(step) + "\n" for step in steps))
        assert replay_module.run(args, stdin=stdin, stdout=io.StringIO()) == 0
        return helpers.collect(out, steps)


def check_replay(which, dtype, steps, sequences, what, slots=4):
    got = run_replay(which, dtype, steps, slots)
    want = plain_logits(which, sequences)
    for name in sequences:
        assert_rows_close(got[name], want[name], dtype, f"{what}/{which}/{name}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_whole_prompts_and_decoded_tails(which, dtype):
    """Each request alone: whole in one step, and most of it in one step with its tail token by token, so that
    prefill and decoding through the cache and the kept state give the same logits.  Sequences of one and two tokens
    (shorter than a convolution) included."""
    sequences = sequences_for(which, [1, 2, 37, 150, 301], seed=10)
    check_replay(which, dtype, helpers.trace_whole(sequences), sequences, "whole")
    check_replay(which, dtype, helpers.trace_tail(sequences, tail=48), sequences, "tail")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_portions_of_every_size(which, dtype):
    """Portions down to two tokens (fewer than the convolution's taps), cut inside pages, key tiles and the runs that
    the recurrence is cut into."""
    sequences = sequences_for(which, [61, 143, 260], seed=20)
    check_replay(which, dtype, helpers.trace_chunks(sequences, seed=1), sequences, "portions")
    check_replay(which, dtype, helpers.trace_chunks(sequences, seed=2, sizes=(2, 2, 17, 64, 3, 130, 2, 31)), sequences,
                 "portions-2")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_mixed_batches_reuse_pages_and_slots(which, dtype):
    """Nine unequal requests through four slots: prompts in portions next to decoded tokens, requests left
    out of steps, pages and state slots handed out again; every request must equal itself alone."""
    sequences = sequences_for(which, [90, 33, 200, 5, 61, 148, 17, 75, 2], seed=30)
    steps = helpers.trace_mixed(sequences, seed=3, live=4, decode_tail=20, max_portion=40)
    assert helpers.peak_tokens(steps) < sum(len(t) for t in sequences.values())
    check_replay(which, dtype, steps, sequences, "mixed")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_requests_decoded_together(dtype):
    """Eleven requests live at once, most of them decoding: batches of single tokens that are padded to shared sizes."""
    sequences = sequences_for("b", [40, 52, 33, 47, 60, 35, 44, 58, 39, 50, 41, 36, 55], seed=90)
    steps = helpers.trace_mixed(sequences, seed=8, live=11, decode_tail=26, max_portion=40)
    check_replay("b", dtype, steps, sequences, "many", slots=11)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["e", "f", "w"])
def test_models_of_one_kind_of_layer(which, dtype):
    sequences = sequences_for(which, [70, 3, 131, 29, 64, 1], seed=70)
    check_replay(which, dtype, helpers.trace_whole(sequences), sequences, "whole")
    steps = helpers.trace_mixed(sequences, seed=5, live=4, decode_tail=16, max_portion=30)
    check_replay(which, dtype, steps, sequences, "mixed")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_of_middle_size(dtype):
    """A thousand tokens whole, then unequal requests mixed, at layer sizes where the tensor-core kernels run."""
    sequences = sequences_for("m", [1000, 260, 97, 23, 1], seed=60)
    check_replay("m", dtype, helpers.trace_whole(sequences), sequences, "whole")
    steps = helpers.trace_mixed(sequences, seed=6, live=4, decode_tail=24, max_portion=70)
    check_replay("m", dtype, steps, sequences, "mixed")


@pytest.mark.parametrize("which,count,tail", [("a", 340, 330), ("c", 200, 190)])
def test_long_decoding_float32(which, count, tail):
    """A short prompt, then hundreds of tokens one by one: the recurrent state and the kept rows of the convolutions
    are carried through every step."""
    sequences = sequences_for(which, [count], seed=40)
    check_replay(which, "float32", helpers.trace_tail(sequences, tail=tail), sequences, "long decode")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_in_one_step_and_in_portions(dtype):
    """1,500 tokens: angles of more than a thousand radians, a recurrence cut into many runs, then the tail decoded."""
    which = "b"
    sequences = sequences_for(which, [1500], seed=80)
    wanted = list(range(0, 1500, 97)) + list(range(1460, 1500))
    whole = [{"step": 0, "entries": [{"id": "s0", "tokens": sequences["s0"], "want": wanted}], "end": ["s0"]}]
    got = run_replay(which, dtype, whole)
    want = plain_logits(which, sequences)["s0"][wanted]
    assert_rows_close(got["s0"], want, dtype, "long prompt in one step")
    steps, number, done = [], 0, 0
    for size in [700, 500, 270] + [1] * 30:
        places = [i for i in range(size) if done + i in wanted]
        steps.append({"step": number, "entries": [{"id": "s0", "tokens": sequences["s0"][done:done + size],
                                                   "want": places}], "end": []})
        number, done = number + 1, done + size
    steps[-1]["end"] = ["s0"]
    got = run_replay(which, dtype, steps)
    assert_rows_close(got["s0"], want, dtype, "long prompt in portions")


# ------------------------------------------------------------------ generation through the scheduler
@pytest.mark.parametrize("strategy", ["orca", "sarathi"])
@pytest.mark.parametrize("which", ["a", "c"])
def test_greedy_generation_equals_the_plain_model(which, strategy):
    from pagedserve_b200.engine.engine import generate

    engine = build_engine(which, "float32", strategy=strategy, prefill_chunk_size=7, max_num_seqs=3)
    prompts = list(sequences_for(which, [9, 30, 3, 55, 1], seed=60).values())
    got = generate(engine, prompts, max_new_tokens=12)
    config, tensors = CONFIGS[which][0], _TENSORS[which]
    for prompt, tokens in zip(prompts, got):
        sequence = list(prompt)
        for _ in range(12):
            logits = plain.forward(tensors, config, sequence)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) < 1e-3 * float(logits.abs().max()):
                break                                        # a near tie: either token is a correct greedy choice
            sequence.append(int(logits.argmax()))
        made = len(sequence) - len(prompt)
        assert tokens[:made] == sequence[len(prompt):]
    engine.check_status()


def test_command_line_runs_a_model_folder(capsys):
    from pagedserve_b200.main import main

    assert main(["--model", folder_of("c"), "--dtype", "bfloat16", "--max-new-tokens", "4", "--block-size", "8",
                 "--num-blocks", "64", "--max-batch-size", "2", "--prompt-ids", "1 2 3 4 5"]) == 0
    assert "request 0:" in capsys.readouterr().out
    # a named size with random weights
    assert main(["--model", "suvunex-tiny", "--seed", "3", "--dtype", "float32", "--max-new-tokens", "5",
                 "--num-blocks", "32", "--max-batch-size", "2", "--prompt-ids", "7 8 9"]) == 0
    assert "request 0:" in capsys.readouterr().out


# ------------------------------------------------------------------ each part alone
def make_ctx(engine, entries):
    from pagedserve_b200.engine.batch import StepEntry

    ctx = engine.runner.prepare([StepEntry(*entry) for entry in entries])
    engine.runner.begin(ctx)
    ctx.shared = {}
    return ctx


def layer_context(engine, index):
    from pagedserve_b200.parts.base import LayerContext

    entry = engine.spec.schedule[index]
    layer = LayerContext(entry.layer, entry.cache_layer, engine.model.positions)
    cache = engine.cache
    group_index = cache.group_of_layer.get(entry.cache_layer)
    if group_index is not None:
        group = cache.groups[group_index]
        layer.k_pool, layer.v_pool = group.layer_views(entry.cache_layer)
        layer.page_stride, layer.page_size = group.page_stride, group.page_size
        layer.pool, layer.pool_layer = group.pool, group.cache_layers.index(entry.cache_layer)
        layer.block_table = cache.slots.table_views[group_index]
    layer.state = cache.state.get(entry.cache_layer)
    return engine.model.blocks[entry.layer], layer


def mixer_share(block, layer):
    """``layer`` as the block hands it to its mixer: without the convolution's rows in front of the state."""
    from pagedserve_b200.parts.parallel import padded, state_share

    at = padded(block.kept)
    if layer.state is None or not block.kept or layer.state.shape[1] <= at:
        return layer
    return state_share(layer, at, layer.state.shape[1] - at)


def run_in_portions(engine, index, fed, tokens, cuts, run, name="x", others=()):
    """``run(block, layer, rows, ctx) -> [T, W] results`` over ``fed`` in portions ``cuts`` (so that later ones start
    from pages, state and kept rows).  ``others``: (name, token) of requests whose single tokens ride in the last
    portion's step."""
    block, layer = layer_context(engine, index)
    result = torch.zeros(fed.shape[0], fed.shape[1], dtype=torch.float32, device=DEV)
    for number, (lo, hi) in enumerate(zip(cuts[:-1], cuts[1:])):
        entries = [(name, tokens[lo:hi], [])]
        rows = fed[lo:hi]
        beside = others if number == len(cuts) - 2 else ()
        if beside:
            entries = [(other, [token], []) for other, token in beside] + entries
            g = torch.Generator().manual_seed(number)
            rows = torch.cat([torch.randn(len(beside), fed.shape[1], generator=g).to(fed.dtype), rows])
        ctx = make_ctx(engine, entries)
        result[lo:hi] = run(block, layer, rows.to(DEV).contiguous(), ctx)[len(beside):]
        engine.cache.commit_many([entry[0] for entry in entries])
    engine.cache.free(name)
    return result


def run_mixer(block, layer, rows, ctx):
    out = torch.zeros(rows.shape, dtype=torch.float32, device=DEV)
    block.mixer.forward(rows, out, ctx, mixer_share(block, layer))
    return out * block.mixer.output_scale


def run_layer(block, layer, rows, ctx):
    """The whole layer on residual rows."""
    carrier = block.begin(rows.float().clone(), ctx)
    block.forward(carrier, ctx, layer)
    rows = block.end(carrier, ctx)
    assert float(carrier.y.abs().max()) == 0.0                       # ready for the next sublayer
    return rows


def plain_mixer(which, index, fed):
    config, tensors = CONFIGS[which][0], _TENSORS[which]
    entry = config["layers"][index]
    tensors = {name: t.double() for name, t in tensors.items() if name.startswith(f"l{index}.")}
    mix = plain.parallel_mixer if entry["type"] == "parallel" else plain.talking_attention
    return mix(tensors, f"l{index}.mix.", entry["mixer"], fed, torch.arange(fed.shape[0]), config["norm"]["eps"])


def plain_layer(which, index, x):
    config, eps = CONFIGS[which][0], CONFIGS[which][0]["norm"]["eps"]
    p = f"l{index}."
    t = lambda name: _TENSORS[which][p + name].double()
    h = plain.with_convolution(plain.rms_norm(x, t("norm1"), eps), t("canon1"))
    x = x + t("ls1") * plain.rms_norm(plain_mixer(which, index, h), t("norm1b"), eps)
    if config["layers"][index]["mlp"] is not None:
        tensors = {name: value.double() for name, value in _TENSORS[which].items()}
        y = plain.gated_ff(tensors, p + "mlp.", plain.rms_norm(x, t("norm2"), eps))
        x = x + t("ls2") * plain.rms_norm(y, t("norm2b"), eps)
    return x


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-6), ("bfloat16", 2.5e-2)])
@pytest.mark.parametrize("which", ["a", "b", "c", "d"])
def test_each_part_alone(which, dtype, tol):
    """Every mixer, every whole layer, the feed-forward, the embedding and the head, each fed with the plain
    implementation's own values.  Mixers and layers run a prompt in three portions (the last of two tokens), so the
    later ones start from pages, state and kept rows."""
    engine = build_engine(which, dtype)
    config, tensors = CONFIGS[which][0], _TENSORS[which]
    eps, compute = config["norm"]["eps"], engine.dtype
    count, cuts = 45, [0, 29, 43, 45]
    tokens = helpers.random_tokens(config["vocab"], count, seed=9)
    g = torch.Generator().manual_seed(5)
    stream = torch.randn(count, config["width"], generator=g, dtype=torch.float64) * 2.0
    for index, entry in enumerate(config["layers"]):
        fed = (stream * 0.5).to(compute)
        got = run_in_portions(engine, index, fed, tokens, cuts, run_mixer)
        assert rel_err(got, plain_mixer(which, index, fed.double())) < tol, (which, index, entry["type"])
        rows = stream.float()
        got = run_in_portions(engine, index, rows, tokens, cuts, run_layer)
        assert rel_err(got, plain_layer(which, index, rows.double())) < tol, (which, index, "layer")
        if entry["mlp"] is not None:
            double = {name: value.double() for name, value in tensors.items()}
            residual = torch.zeros(count, config["width"], dtype=torch.float32, device=DEV)
            engine.model.blocks[index].feed_forward.forward(fed.to(DEV), residual, None)
            assert rel_err(residual, plain.gated_ff(double, f"l{index}.mlp.", fed.double())) < tol, (which, index, "mlp")
    # the embedding times its constant, the model's norm on chosen rows, and the head times its constant
    ctx = make_ctx(engine, [("z", tokens, [0, 7, 44])])
    embedded = engine.model.embedding.forward(ctx, engine.model.positions)
    assert rel_err(embedded, tensors["embed"].double()[tokens] * config["embedding"]["scale"]) < 1e-6
    picked = engine.model.final_norm.forward(stream.float().to(DEV), rows=ctx.logit_rows)
    logits = engine.model.head.forward(picked, engine.model.embedding)
    want = (plain.rms_norm(stream, tensors["final.norm"].double(), eps)[[0, 7, 44]] @ tensors["head"].double().T
            * config["logit_scale"])
    assert rel_err(logits, want) < tol
    engine.cache.rollback("z")
    engine.cache.free("z")
    engine.check_status()


# ------------------------------------------------------------------ the recurrence alone
def recurrence_case(heads, dk, dv, rank, lengths, seed, dtype, tau=4.0):
    g = torch.Generator().manual_seed(seed)
    total = sum(lengths)
    gap = 3 if dk % 8 else 0                                            # odd places: the number-by-number loads
    widths = [heads * dk, heads * dk, heads * dv, heads * dv, rank]
    offsets, at = [], gap
    for width in widths:
        offsets.append(at)
        at += width
    rows = torch.randn(total, at + (-at % 8 if not gap else 1), generator=g).to(dtype)
    a2 = torch.randn(heads * dk, rank, generator=g) * rank ** -0.5
    bias = 1.5 * torch.randn(heads * dk, generator=g)
    gain = 1.0 + 0.2 * torch.randn(dv, generator=g)
    items = len(lengths)
    state = torch.randn(items + 1, heads * dk * dv + 8, generator=g)
    starts = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
    slots = torch.randperm(items, generator=g).to(torch.int32)
    eps, out_scale, q_scale = 1e-4, 0.7, dk ** -0.5
    part = lambda i: rows[:, offsets[i]:offsets[i] + widths[i]].double()
    q, k = part(0).reshape(total, heads, dk) * q_scale, part(1).reshape(total, heads, dk)
    v, gate = part(2).reshape(total, heads, dv), part(3).reshape(total, heads, dv)
    alpha = torch.sigmoid(part(4) @ a2.double().T + bias.double()).pow(1.0 / tau).reshape(total, heads, dk)
    want = torch.empty(total, heads, dv, dtype=torch.float64)
    final = state.double().clone()
    for item, (lo, hi) in enumerate(zip(starts[:-1], starts[1:])):
        S = state[slots[item], :heads * dk * dv].double().reshape(heads, dk, dv)
        for t in range(lo, hi):
            S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            want[t] = torch.einsum("hd,hde->he", q[t], S)
        final[slots[item], :heads * dk * dv] = S.reshape(-1)
    want = plain.rms_norm(want, gain.double(), eps) * gate * torch.sigmoid(gate) * out_scale
    short = sum(1 for n in lengths if n < 16)
    ctx = SimpleNamespace(max_q_len=max(lengths), q_start=torch.from_numpy(starts).to(DEV), item_slot=slots.to(DEV),
                          num_items=items, num_short_items=short, single_tokens=max(lengths) == 1)

    def run(ops, segments=None):
        kept = state.to(DEV)
        out = torch.full((total, heads * dv + 5), 7.0, dtype=dtype, device=DEV)
        ops.gla_recurrence(rows.to(DEV), offsets, a2.to(DEV), bias.to(DEV), tau, q_scale, gain.to(DEV), eps, out_scale, kept,
                           ctx, out[:, :heads * dv], heads, dk, dv, segments=segments)
        assert bool((out[:, heads * dv:] == 7.0).all())
        return out[:, :heads * dv], kept

    return run, want.reshape(total, heads * dv), final


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dk,dv,rank,lengths", [
    (3, 16, 24, 5, [1, 1, 1]), (2, 64, 64, 16, [1, 2, 15, 40, 200]), (1, 128, 128, 33, [3, 130]), (4, 20, 36, 1, [7, 17, 333]),
    (2, 40, 100, 70, [100]), (1, 96, 32, 8, [1, 64, 65]), (2, 8, 128, 12, [50, 31]), (2, 144, 160, 16, [1, 20]),
    (5, 10, 14, 16, [16, 16, 150]), (2, 64, 128, 16, [1] * 5), (3, 128, 64, 70, [1, 1]), (4, 10, 14, 3, [1] * 4),
    (2, 32, 96, 9, [1] * 3)])
def test_the_recurrence_alone(heads, dk, dv, rank, lengths, dtype):
    """Entries of unequal length (short ones first) from states that are not zero, in one piece and cut into runs that
    are worked on side by side (also into more runs than the entry has chunks), equal the plain loop; the state that is
    left is where a next step starts from."""
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(dtype)
    run, want, final = recurrence_case(heads, dk, dv, rank, lengths, seed=heads + dk + dv, dtype=dtype)
    for segments in (1, 2, 5, 64, None):
        out, kept = run(ops, segments)
        assert rel_err(out, want) < (1e-5 if dtype == torch.float32 else 6e-3), segments
        assert rel_err(kept, final) < 5e-6, segments


def test_decays_at_both_ends():
    """Decay arguments of +-60: alpha is one and zero to the last bit, and nothing overflows on the way."""
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(torch.float32)
    heads, dk, dv, total = 1, 16, 16, 40
    g = torch.Generator().manual_seed(0)
    rows = torch.randn(total, 4 * 16 + 8, generator=g)
    bias = torch.where(torch.arange(dk) % 2 == 0, 60.0, -60.0)
    a2 = torch.zeros(dk, 1)
    ctx = SimpleNamespace(max_q_len=total, q_start=torch.tensor([0, total], dtype=torch.int32, device=DEV),
                          item_slot=torch.zeros(1, dtype=torch.int32, device=DEV), num_items=1, num_short_items=0)
    for tau in (0.25, 16.0):
        alpha = torch.sigmoid(bias.double()).pow(1.0 / tau)
        S, want = torch.zeros(dk, dv, dtype=torch.float64), []
        for t in range(total):
            S = alpha[:, None] * S + rows[t, 16:32].double()[:, None] * rows[t, 32:48].double()[None, :]
            want.append(rows[t, :16].double() @ S)
        gate = rows[:, 48:64].double()
        want = plain.unit_rms(torch.stack(want), 1e-6) * gate * torch.sigmoid(gate)
        state = torch.zeros(1, dk * dv, device=DEV)
        out = torch.empty(total, dv, device=DEV)
        ops.gla_recurrence(rows.to(DEV), (0, 16, 32, 48, 64), a2.to(DEV), bias.to(DEV), tau, 1.0, torch.ones(dv, device=DEV),
                           1e-6, 1.0, state, ctx, out, heads, dk, dv, segments=3)
        assert rel_err(out, want) < 1e-5 and rel_err(state.view(dk, dv), S) < 1e-5


# ------------------------------------------------------------------ the convolution, the close of a sublayer, the mixed heads
@pytest.mark.parametrize("width", [40, 37])
@pytest.mark.parametrize("taps,lengths", [(1, [5, 1]), (2, [1, 1, 9]), (3, [2, 1, 40, 1]), (4, [1, 2, 3, 200]), (3, [1, 1, 1]),
                                          (7, [3, 3, 1])])
def test_the_convolution_on_scaled_rows(taps, lengths, width):
    """A factor per row that stands for the row's norm, entries shorter and longer than the convolution, three steps in
    a row: each starts from the rows that the one before kept (steps of single tokens keep theirs in the same kernel)."""
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(torch.float32)
    g = torch.Generator().manual_seed(taps)
    weight = torch.randn(width, taps, generator=g)
    bare = weight.clone()
    bare[:, -1] -= 1.0                                                # h + conv(h) is a convolution itself
    items = len(lengths)
    slots = torch.randperm(items, generator=g).to(torch.int32)
    state = torch.zeros(items + 1, (taps - 1) * width + 12, device=DEV)
    kept = state[:, :(taps - 1) * width] if taps > 1 else None       # a share of a longer row
    history = [torch.zeros(0, width, dtype=torch.float64) for _ in lengths]
    for step in range(4):
        counts = [1] * items if step == 2 else lengths if step % 2 == 0 else lengths[::-1]
        starts = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
        u = torch.randn(int(starts[-1]), width, generator=g)
        scale = 0.5 + torch.rand(int(starts[-1]), generator=g)
        token_item = torch.repeat_interleave(torch.arange(items), torch.tensor(counts)).to(torch.int32)
        want = torch.empty(u.shape, dtype=torch.float64)
        for item, (lo, hi) in enumerate(zip(starts[:-1], starts[1:])):
            before = history[item].shape[0]
            history[item] = torch.cat([history[item], u[lo:hi].double() * scale[lo:hi, None].double()])
            want[lo:hi] = plain.with_convolution(history[item], bare.double())[before:]
        ctx = SimpleNamespace(token_item=token_item.to(DEV), q_start=torch.from_numpy(starts).to(DEV),
                              item_slot=slots.to(DEV), num_items=items, single_tokens=max(counts) == 1)
        out = torch.empty(u.shape, device=DEV)
        ops.short_conv(u.to(DEV), weight.to(DEV), taps, width, kept, ctx, out, row_scale=scale.to(DEV))
        assert rel_err(out, want) < 3e-6, (taps, step)
    assert float(state[:, (taps - 1) * width:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width", [(1, 64), (37, 50), (9, 1024), (5, 2056), (3, 9000), (6, 36)])
def test_the_close_of_a_sublayer(rows, width, dtype):
    from pagedserve_b200.kernels.ops import Ops

    compute = torch.float32 if dtype == "float32" else torch.bfloat16
    ops = Ops(compute)
    g = torch.Generator().manual_seed(width)
    x, y = torch.randn(rows, width, generator=g) * 3.0, torch.randn(rows, width, generator=g) * 0.01
    gain, next_gain = torch.randn(width, generator=g), 1.0 + 0.3 * torch.randn(width, generator=g)
    eps, y_scale = 1e-4, -0.6                                         # eps shows beside rows this small
    summed = x.double() + plain.rms_norm(y_scale * y.double(), gain.double(), eps)
    xs, ys = x.to(DEV), y.to(DEV)
    out = torch.empty(rows, width, dtype=compute, device=DEV)
    scale = torch.empty(rows, device=DEV)
    ops.sandwich_close(ys, xs, gain.to(DEV), y_scale, eps, next_gain.to(DEV), out, scale)
    assert rel_err(xs, summed) < 2e-6 and float(ys.abs().max()) == 0.0
    assert rel_err(out, plain.rms_norm(summed, next_gain.double(), eps)) < (3e-6 if dtype == "float32" else 5e-3)
    assert rel_err(scale, 1.0 / torch.sqrt((summed * summed).mean(-1) + eps)) < 2e-6
    ys = y.to(DEV)                                                    # the opening: nothing is added
    ops.sandwich_close(ys, xs, None, 1.0, eps, row_scale=scale)
    assert float(ys.abs().max()) == 0.0 and rel_err(xs, summed) < 2e-6


@pytest.mark.parametrize("taps", [1, 2, 3, 4])
@pytest.mark.parametrize("rows,width", [(1, 64), (6, 1024), (3, 2052)])
def test_the_close_and_the_next_convolution_in_one_kernel(rows, width, taps):
    """Single tokens: the fused kernel leaves what the close and the convolution one after the other leave, the kept rows
    included, twice in a row."""
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(torch.bfloat16)
    g = torch.Generator().manual_seed(width + taps)
    gain, weight = torch.randn(width, generator=g).to(DEV), torch.randn(width, taps, generator=g).to(DEV)
    slots = torch.randperm(rows, generator=g).to(torch.int32).to(DEV)
    state = torch.randn(rows + 1, (taps - 1) * width + 4, generator=g).to(DEV)
    ctx = SimpleNamespace(token_item=torch.arange(rows, dtype=torch.int32, device=DEV), item_slot=slots, num_items=rows,
                          q_start=torch.arange(rows + 1, dtype=torch.int32, device=DEV), single_tokens=True)
    kept_a, kept_b = state.clone(), state.clone()
    share = lambda kept: kept[:, :(taps - 1) * width] if taps > 1 else None
    for factor in (0.7, None):
        x, y = torch.randn(rows, width, generator=g).to(DEV), torch.randn(rows, width, generator=g).to(DEV)
        xa, ya, xb, yb = x.clone(), y.clone(), x.clone(), y.clone()
        own = gain if factor is not None else None
        scale = torch.empty(rows, device=DEV)
        a, b = (torch.empty(rows, width, dtype=torch.bfloat16, device=DEV) for _ in range(2))
        ops.sandwich_close(ya, xa, own, factor or 1.0, 1e-5, row_scale=scale)
        ops.short_conv(xa, weight, taps, width, share(kept_a), ctx, a, row_scale=scale)
        assert ops.close_conv_ok(yb, weight, taps, share(kept_b))
        ops.sandwich_close_conv(yb, xb, own, factor or 1.0, 1e-5, weight, taps, share(kept_b), ctx, b)
        assert rel_err(xb, xa.cpu()) < 1e-6 and float(yb.abs().max()) == 0.0
        assert rel_err(b.float(), a.float().cpu()) < 5e-3 and rel_err(kept_b, kept_a.cpu()) < 1e-6


def paged_case(tokens, positions, kv_heads, dim, page, seed, dtype):
    """A pool of keys and values in shuffled pages and one block-table row per token's request."""
    g = torch.Generator().manual_seed(seed)
    pages = max(positions) // page + 1
    pool = torch.randn(pages + 3, 1, 2, kv_heads, page, dim, generator=g).to(dtype)
    table = (torch.randperm(pages + 3, generator=g)[:pages]).to(torch.int32)[None]
    keys = pool[table[0].long(), 0, 0].permute(1, 0, 2, 3).reshape(kv_heads, pages * page, dim).double()
    values = pool[table[0].long(), 0, 1].permute(1, 0, 2, 3).reshape(kv_heads, pages * page, dim).double()
    return pool.to(DEV), table.to(DEV), keys, values


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,page", [(4, 2, 16, 16), (6, 3, 48, 8), (8, 8, 64, 16), (4, 2, 128, 32), (5, 1, 64, 16),
                                                     (6, 2, 20, 16), (12, 4, 96, 16), (20, 4, 32, 16), (16, 4, 64, 16),
                                                     (16, 8, 32, 8), (12, 3, 64, 16)])
@pytest.mark.parametrize("form", ["single", "portion"])
def test_every_query_head_meets_every_value_head(heads, kv_heads, dim, page, form, dtype):
    """Attention with all values and the mixing kernel against the equations: single tokens at many positions, and a
    prompt portion behind cached keys; learned sinks; one key that stands out for one head."""
    from pagedserve_b200.kernels import tensorcore
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(dtype)
    g = torch.Generator().manual_seed(heads * dim + page)
    positions = [0, 1, 17, 63, 64, 130, 255, 256, 300, 511] if form == "single" else list(range(90, 347))
    count = len(positions)
    pool, table, keys, values = paged_case(count, positions, kv_heads, dim, page, seed=dim, dtype=dtype)
    q = torch.randn(count, heads * dim, generator=g)
    q[:, :dim] = keys[0, 0].float() * 0.4                             # key 0 draws head 0 wherever it is
    q = q.to(dtype)
    sink, talk = torch.randn(heads, generator=g), torch.eye(heads) + 0.4 * torch.randn(heads, heads, generator=g)
    scale = dim ** -0.5
    group = torch.arange(heads) // (heads // kv_heads)
    at = torch.tensor(positions)
    scores = torch.einsum("thd,hjd->htj", q.double().reshape(count, heads, dim), keys[group]) * scale
    scores = scores.masked_fill(torch.arange(keys.shape[1])[None, None, :] > at[None, :, None], float("-inf"))
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink.double()[:, None, None])
    weights = torch.exp(scores - top)
    weights = weights / (weights.sum(-1, keepdim=True) + torch.exp(sink.double()[:, None, None] - top))
    want_all = torch.einsum("htj,ejd->thed", weights, values)
    mixed = torch.einsum("hg,gtj->htj", talk.double(), weights)
    want = torch.einsum("htj,hjd->thd", mixed, values[group]).reshape(count, heads * dim)

    single = form == "single"
    layer = SimpleNamespace(k_pool=pool[:, 0, 0], v_pool=pool[:, 0, 1], page_stride=pool.stride(0), page_size=page, pool=pool,
                            pool_layer=0, block_table=table)
    zeros = torch.zeros(count, dtype=torch.int32, device=DEV)
    place = torch.tensor(positions, dtype=torch.int32, device=DEV)
    items = count if single else 1
    ctx = SimpleNamespace(num_tokens=count, num_items=items, num_short_items=items if single else 0,
                          num_short_tokens=count if single else 0, num_long_blocks=0 if single else -(-count // 64),
                          token_item=torch.arange(count, dtype=torch.int32, device=DEV) if single else zeros, token_slot=zeros,
                          positions=place, max_kv_len=max(positions) + 1, status=ops.status_flag(DEV),
                          q_start=torch.tensor(list(range(count + 1)) if single else [0, count], dtype=torch.int32, device=DEV),
                          kv_len=place + 1 if single else torch.tensor([positions[-1] + 1], dtype=torch.int32, device=DEV),
                          item_slot=torch.zeros(items, dtype=torch.int32, device=DEV))
    q = q.to(DEV)
    tol = 5e-6 if dtype == torch.float32 else 1.2e-2
    wide = torch.full((count, heads * dim + 8), 9.0, dtype=dtype, device=DEV)
    ops.attention(q, None, None, wide[:, :heads * dim], ctx, layer, heads, kv_heads, dim, None, scale, write_cache=False,
                  sink=sink.to(DEV), mix=talk.to(DEV).contiguous())
    assert rel_err(wide[:, :heads * dim], want) < tol and bool((wide[:, heads * dim:] == 9.0).all())
    # the two steps alone, on the kernel that takes every head size
    every = torch.full((count, heads * kv_heads * dim), 9.0, dtype=dtype, device=DEV)
    ops.paged_attention_simt(q, every, layer.k_pool, layer.v_pool, layer.page_stride, zeros, place, table, heads, kv_heads, dim,
                             page, None, scale, sink=sink.to(DEV), all_values=True)
    assert rel_err(every, want_all.reshape(count, -1)) < tol
    out = torch.empty(count, heads * dim, dtype=dtype, device=DEV)
    ops.head_mix(every, talk.to(DEV).contiguous(), out, heads, kv_heads, dim)
    assert rel_err(out, want) < tol
    assert int(ops.status_flag(DEV).item()) == 0


@pytest.mark.parametrize("heads,kv_heads,dim,page,window,softcap,with_sink", [
    (8, 2, 64, 16, None, None, True), (16, 1, 128, 16, None, None, False), (12, 3, 48, 8, 100, None, True),
    (20, 4, 96, 32, None, 20.0, True), (4, 1, 16, 16, -70, None, False), (32, 2, 32, 16, 33, None, True),
    (7, 7, 112, 16, None, None, True), (10, 2, 80, 64, None, None, False)])
@pytest.mark.parametrize("splits", [1, 2, 8, None])
def test_heads_of_a_group_as_rows(heads, kv_heads, dim, page, window, softcap, with_sink, splits):
    """Single tokens with the heads of a group as the rows of a tile against the CUDA-core kernel: positions at tile and
    page borders, windows and chunked masks, capped scores, sinks, and more CTAs than some tokens have key tiles."""
    from pagedserve_b200.kernels.ops import Ops

    ops = Ops(torch.bfloat16)
    positions = [0, 1, 15, 16, 31, 63, 64, 130, 255, 256, 299, 700]
    count = len(positions)
    pool, table, _, _ = paged_case(count, positions, kv_heads, dim, page, seed=dim + heads, dtype=torch.bfloat16)
    g = torch.Generator().manual_seed(heads)
    q = (torch.randn(count, heads * dim + 16, generator=g)).to(torch.bfloat16).to(DEV)[:, :heads * dim]
    sink = torch.randn(heads, generator=g).to(DEV) if with_sink else None
    zeros, place = torch.zeros(count, dtype=torch.int32, device=DEV), torch.tensor(positions, dtype=torch.int32, device=DEV)
    own = torch.arange(count, dtype=torch.int32, device=DEV)
    want, got = torch.empty(count, heads * dim, dtype=torch.bfloat16, device=DEV), torch.empty(count, heads * dim,
                                                                                           dtype=torch.bfloat16, device=DEV)
    args = (pool[:, 0, 0], pool[:, 0, 1], pool.stride(0))
    ops.paged_attention_simt(q, want, *args, zeros, place, table, heads, kv_heads, dim, page, window, dim ** -0.5, softcap, sink)
    ops.attention_rows(q, got, *args, own, place, table, heads, kv_heads, dim, page, window, dim ** -0.5, max(positions) + 1,
                       q_start=torch.arange(count + 1, dtype=torch.int32, device=DEV), kv_len=place + 1, token_row=zeros,
                       softcap=softcap, sink=sink, splits=splits)
    assert rel_err(got, want.float().cpu()) < 1.2e-2


# ------------------------------------------------------------------ a key that stands out, at page borders and far back
def standing_out(index, key_at, query_at, count, seed):
    """Rows for the mixer of layer ``index`` such that query head 0 at ``query_at`` points straight along the key of key
    head 0 at ``key_at`` as attention meets it.  The norms remove the query's size, so the rows are solved for its
    direction only; steep scales and large query gains make the key decide."""
    config, tensors = CONFIGS["s"][0], _TENSORS["s"]
    entry = config["layers"][index]
    eps = config["norm"]["eps"]
    left = entry["type"] == "parallel"
    m, names = (entry["mixer"]["left"], "left.") if left else (entry["mixer"], "")
    g = torch.Generator().manual_seed(seed)
    rows = torch.randn(count, config["width"], generator=g, dtype=torch.float64)
    t = lambda name: tensors[f"l{index}.mix.{names}{name}"].double()
    where = torch.tensor([key_at - query_at])
    d = m["dim"]
    key = (rows[key_at] @ t("k").T + t("k.b"))[:d][None, None]
    key = plain.unit_rms(key, eps) if left else plain.rms_norm(key, t("k.norm"), eps)
    target = plain.rotate_halves(key, where, m["rot"])[0, 0]
    wanted = 6.0 * (target if left else target / t("q.norm")) - t("q.b")[:d]
    rows[query_at] = torch.linalg.lstsq(t("q")[:d], wanted[:, None]).solution[:, 0]
    return rows


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-5), ("bfloat16", 2.5e-2)])
@pytest.mark.parametrize("index", [0, 1, 2, 3, 4])
def test_a_key_that_stands_out_at_page_borders_and_far_back(index, dtype, tol):
    """One query made to point at one key: at the sequence's first token, at the query itself, on both sides of page and
    tile borders and hundreds of tokens back; in a prompt in one step, in two portions cut between the two tokens, with
    the query decoded alone, and decoded among single tokens of other requests."""
    from pagedserve_b200.engine.batch import StepEntry

    engine = build_engine("s", dtype)
    config = CONFIGS["s"][0]
    count = 300
    tokens = helpers.random_tokens(config["vocab"], count, seed=2)
    for other in ("p", "q", "r"):                        # three other requests hold state and pages of their own
        engine.step([StepEntry(other, helpers.random_tokens(config["vocab"], 20, seed=ord(other)), [])])
    for query_at, key_at in ((299, 0), (299, 3), (150, 1), (255, 16), (256, 255), (272, 271), (17, 15), (128, 127), (40, 40)):
        fed = standing_out(index, key_at, query_at, count, seed=query_at + key_at).to(engine.dtype)
        want = plain_mixer("s", index, fed.double())
        if key_at != query_at:
            # the key decides the row: with another key in its place the plain result is another one altogether
            changed = fed.double().clone()
            changed[key_at] = 0.0
            moved = plain_mixer("s", index, changed)[query_at]
            assert float((moved - want[query_at]).abs().max()) > 0.05 * float(want[query_at].abs().max())
        alone = [0, query_at, query_at + 1, count] if query_at + 1 < count else [0, query_at, count]
        for cuts, others in (([0, count], ()), ([0, key_at + 1, count] if key_at < query_at else [0, 7, count], ()),
                             (alone, ()), (alone[:-1] if len(alone) == 4 else alone, (("p", 1), ("q", 2), ("r", 3)))):
            got = run_in_portions(engine, index, fed[:cuts[-1]], tokens, cuts, run_mixer, others=others)
            assert rel_err(got[query_at], want[query_at]) < tol, (index, query_at, key_at, cuts)
            assert rel_err(got, want[:cuts[-1]]) < tol, (index, query_at, key_at, cuts)
    engine.check_status()


def test_a_sink_and_the_one_in_the_denominator_show():
    """A sequence's first token sees one key only: without a sink its weight would be one whatever its score.  The
    engine's row must carry the weight e^s / (e^s + e^sink), and the plain rows with and without differ by far more than
    the tolerance."""
    for index in (0, 2):
        engine = build_engine("s", "float32")
        config = CONFIGS["s"][0]
        fed = torch.randn(3, config["width"], generator=torch.Generator().manual_seed(index), dtype=torch.float64)
        got = run_in_portions(engine, index, fed.float(), [1, 2, 3], [0, 1, 3], run_mixer)
        assert rel_err(got, plain_mixer("s", index, fed.float().double())) < 1e-5
        original = plain.causal_softmax
        try:
            plain.causal_softmax = lambda scores, extra: original(scores, torch.full_like(extra.double(), -1e9))
            bare = plain_mixer("s", index, fed.float().double())
        finally:
            plain.causal_softmax = original
        assert rel_err(got, bare) > 0.05
