"""Benchmark of the engine's decode step (and prefill) for GPT-2 124M layer sizes, random weights.

    python bench.py --gpus 1 --steps K --warmup W            # this engine
    python bench.py --impl reference --gpus 1 ...            # the unmodified reference, if installed

A "step" is one decode step of the whole batch.  The default run: layer sizes of GPT-2 124M,
bfloat16, batch 8, 512-token prompts of uniform-random token ids, then K decode steps.

value     decoded tokens per second over K steps timed on the device (CUDA events): the captured
          decode step replayed K times, sampling and token feedback on the device.
e2e       the same through the Python entry point (``Scheduler.step``): every step the host builds
          the batch, copies it from pinned memory to the device and reads the sampled tokens back.
          (The scheduler launches the next step of an unchanged batch behind the running one: that
          step's token ids are the ones the device fed back, every other input is uploaded.)
prefill   one step of 2,048 prompt tokens (2 prompts of 1,024).
roofline  bytes the decode step has to read (every weight once + the cache of the live requests)
          divided by its time, against the measured copy bandwidth.
points    decode tokens per second at batch 1 and 64.
"""

from __future__ import annotations

import argparse
import json
import math
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def load_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as handle:
                data = json.load(handle)
            flat = {}

            def walk(node):
                if isinstance(node, dict):
                    for key, value in node.items():
                        if isinstance(value, (int, float)) and key not in flat:
                            flat[key] = float(value)
                        else:
                            walk(value)

            walk(data)
            if "hbm_gbs" in flat and "bf16_tflops" in flat:
                return {"hbm_gbs": flat["hbm_gbs"], "bf16_tflops": flat["bf16_tflops"],
                        "bf16_tflops_sustained": flat.get("bf16_tflops_sustained"), "source": "measured"}
        except Exception:
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self._stop = threading.Event()
        self._thread = None

    def _run(self):
        while not self._stop.is_set():
            try:
                out = subprocess.run(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                      "--format=csv,noheader,nounits"], capture_output=True, text=True, timeout=5)
                parts = [p.strip() for p in out.stdout.strip().splitlines()[0].split(",")]
                self.samples.append(parts)
            except Exception:
                pass
            self._stop.wait(0.2)

    def __enter__(self):
        self._thread = threading.Thread(target=self._run, daemon=True)
        self._thread.start()
        return self

    def __exit__(self, *exc):
        self._stop.set()
        self._thread.join(timeout=6)

    def summary(self):
        clocks = [int(s[0]) for s in self.samples if s and s[0].isdigit()]
        maxes = [int(s[1]) for s in self.samples if len(s) > 1 and s[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({names[i] for s in self.samples for i in range(4)
                          if len(s) > 2 + i and s[2 + i].lower().startswith("active")})
        return {"sm_mhz": int(statistics.median(clocks)) if clocks else None,
                "sm_max_mhz": max(maxes) if maxes else None, "reasons": reasons, "samples": len(clocks)}


def _reference_tree():
    """The folder that holds the unmodified reference (its ``main.py`` and ``src/``), or (None, why).

    jainalphin/pagedserve is a script tree without setup.py or pyproject.toml, so ``pip install --target
    baseline/_ref`` refuses it; a plain copy of the checkout stands in its place.  Where the copy is missing
    and ``PAGEDSERVE_REFERENCE_SRC`` names a checkout, the copy is made now."""
    ref = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isfile(os.path.join(ref, "src", "model", "paged_decoder.py")):
        source = os.environ.get("PAGEDSERVE_REFERENCE_SRC", "")
        if not os.path.isfile(os.path.join(source, "src", "model", "paged_decoder.py")):
            return None, ("baseline/_ref holds no copy of jainalphin/pagedserve (pip refuses the tree: neither "
                          "setup.py nor pyproject.toml) and PAGEDSERVE_REFERENCE_SRC names no checkout")
        import shutil

        os.makedirs(ref, exist_ok=True)
        shutil.copytree(os.path.join(source, "src"), os.path.join(ref, "src"), dirs_exist_ok=True)
        shutil.copy(os.path.join(source, "main.py"), os.path.join(ref, "main.py"))
    return ref, None


def reference_arm(args):
    """The same measurements on the unmodified reference: its own ``PagedDecoderLM`` with random weights at the
    named layer sizes, its ``KVCacheManager``, ``PagedAttention`` and ``ContinuousBatchScheduler``
    (reference: main.py:104-116, 215-254; benchmark.py:106-128; src/scheduler/orca_scheduler.py:85-117,
    221-303), driven through ``add_token_request`` and ``step`` with the same seeded prompts, warm-up and step
    count as this engine's arm.  Nothing of ``pagedserve_b200`` but the table of layer sizes is imported."""
    ref, why = _reference_tree()
    if ref is None:
        print(json.dumps({"impl": "reference", "unavailable": why}))
        return 0
    try:
        result = _run_reference(args, ref)
    except Exception as error:                                    # the arm must not take the driver down
        message = " ".join(f"{type(error).__name__}: {error}".split())[:300]
        print(json.dumps({"impl": "reference", "unavailable": f"the reference raised: {message}"}))
        return 0
    print(json.dumps(result))
    return 0


def _run_reference(args, ref):
    import importlib.util

    import numpy as np
    import torch

    from pagedserve_b200.config.gpt2 import NAMED_CONFIGS          # layer sizes only: plain Python, no kernels

    sys.path.insert(0, ref)
    from src.model.kv_manager import KVCacheManager
    from src.model.paged_attention import PagedAttention
    from src.model.paged_decoder import PagedDecoderLM, TransformerConfig
    from src.scheduler.orca_scheduler import ContinuousBatchScheduler

    sizes = dict(NAMED_CONFIGS[args.model])
    full_layers = sizes["n_layer"]
    if args.layers:
        sizes["n_layer"] = args.layers
    hidden, heads, inner = sizes["n_embd"], sizes["n_head"], sizes["n_inner"] or 4 * sizes["n_embd"]
    context_len, vocab = sizes["n_positions"], sizes["vocab_size"]
    steps, warmup = args.steps, max(args.warmup, 3)
    if args.prompt_len + warmup + steps + 2 > context_len:
        steps = context_len - args.prompt_len - warmup - 2
    dtype = torch.bfloat16 if args.dtype == "bfloat16" else torch.float32
    on_gpu = torch.cuda.is_available()               # without a GPU the arm still runs (a dry run of its host side)
    device = torch.device("cuda" if on_gpu else "cpu")
    backend = "triton" if on_gpu and importlib.util.find_spec("triton") is not None else "torch"

    class DeviceTimer:
        """Milliseconds between ``start`` and ``stop`` on the device (CUDA events); wall clock without a GPU."""

        def start(self):
            if on_gpu:
                self.events = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                self.events[0].record()
            self.began = time.perf_counter()

        def stop(self):
            if on_gpu:
                self.events[1].record()
                torch.cuda.synchronize()
            self.seconds = time.perf_counter() - self.began
            return self.events[0].elapsed_time(self.events[1]) if on_gpu else self.seconds * 1e3
    peaks = load_peaks()

    torch.manual_seed(0)                                           # reference: benchmark.py:106-107
    model = PagedDecoderLM(TransformerConfig(
        vocab_size=vocab, hidden_size=hidden, num_layers=sizes["n_layer"], num_heads=heads,
        head_dim=hidden // heads, mlp_hidden_size=inner, max_sequence_length=context_len,
        activation_function="gelu_tanh", layer_norm_epsilon=sizes["layer_norm_epsilon"],
        tie_word_embeddings=True, lm_head_bias=False))
    model = model.to(device=device, dtype=dtype).eval()            # reference: main.py:133
    model.enable_cuda_graphs = True                                # reference: main.py:193
    max_batch = max(64, args.batch)
    width = 2 if dtype == torch.bfloat16 else 4
    block_bytes = 2 * sizes["n_layer"] * hidden * 16 * width
    cache = KVCacheManager(block_size=16, total_memory=(max_batch * (context_len // 16) + 64) * block_bytes,
                           tensor_dtype=dtype, device=device, num_layers=sizes["n_layer"], num_kv_heads=heads,
                           head_dim=hidden // heads, cache_dtype=dtype)          # reference: main.py:214-223
    attention = PagedAttention(kv_manager=cache, decode_attention_backend=backend)
    rng = np.random.default_rng(0)
    weight_bytes = sum(p.numel() * p.element_size() for name, p in model.named_parameters()
                       if not name.startswith("position_embeddings"))
    kv_bytes_per_token = 2 * sizes["n_layer"] * hidden * width

    def make_scheduler(batch):
        return ContinuousBatchScheduler(model_engine=model, max_batch_size=batch, tokenizer=None, kv_manager=cache,
                                        paged_attn_manager=attention, eos_token_id=None,
                                        scheduling_strategy="orca")

    def measure_decode(batch, k_steps):
        scheduler = make_scheduler(batch)
        for _ in range(batch):
            scheduler.add_token_request(rng.integers(0, vocab, args.prompt_len).tolist(),
                                        max_new_tokens=warmup + k_steps + 2)
        while scheduler.waiting:
            scheduler.step()                                       # the prompts (untimed)
        for _ in range(warmup):
            scheduler.step()
        timer, produced = DeviceTimer(), 0
        with ClockSampler() as clocks:
            timer.start()
            for _ in range(k_steps):
                produced += len(scheduler.step())
            ms = timer.stop()
        seconds = timer.seconds
        _drain(scheduler)
        mean_context = args.prompt_len + warmup + (k_steps + 1) / 2.0
        return {"ms": ms, "tok_s": produced / (ms / 1e3), "e2e_tok_s": produced / seconds,
                "e2e_ms_per_step": seconds * 1e3 / k_steps,
                "bytes_per_step": weight_bytes + batch * mean_context * kv_bytes_per_token,
                "clocks": clocks.summary()}

    def _drain(scheduler):
        while scheduler.waiting or scheduler.active:
            scheduler.step()

    def measure_prefill(tokens_total=2048, repeats=5):
        prompt_len = min(1024, context_len - 1)
        count = max(1, tokens_total // prompt_len)
        times = []
        for repeat in range(repeats + 3):
            scheduler = make_scheduler(count)
            for _ in range(count):
                scheduler.add_token_request(rng.integers(0, vocab, prompt_len).tolist(), max_new_tokens=1)
            timer = DeviceTimer()
            timer.start()
            scheduler.step()                                       # whole prompts in one iteration (Orca)
            elapsed = timer.stop()
            if repeat >= 3:
                times.append(elapsed)
            _drain(scheduler)
        ms = statistics.median(times)
        T = count * prompt_len
        L = sizes["n_layer"]
        gemm = 2.0 * T * L * (4 * hidden * hidden + 2 * hidden * inner) + 2.0 * count * hidden * vocab
        flops = gemm + L * count * 4.0 * hidden * (prompt_len * (prompt_len + 1) / 2.0)
        peak = peaks["bf16_tflops"] * 1e12 if dtype == torch.bfloat16 else 75e12
        return {"value": T / (ms / 1e3), "tokens": T, "ms": ms, "frac": flops / (ms / 1e3) / peak,
                "gflop": flops / 1e9}

    with torch.inference_mode():
        main_run = measure_decode(args.batch, steps)
        result = {
            "metric": "decode tok/s at batch 1/8/64; prefill tok/s at 2,048 tokens (GPT-2 124M)",
            "value": main_run["tok_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
            "ms_per_step": main_run["ms"] / steps, "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16" if dtype == torch.bfloat16 else "fp32", "data": "synthetic",
            "impl": "reference", "decode_attention_backend": backend,
            "config": {
                "model": args.model, "weights": "random(torch.manual_seed(0))", "n_layer": sizes["n_layer"],
                "n_layer_full": full_layers, "n_embd": hidden, "n_head": heads, "n_inner": inner,
                "vocab_size": vocab, "n_positions": context_len, "global_batch": args.batch,
                "seq_len": context_len, "prompt_len": args.prompt_len, "generated": steps, "block_size": 16,
                "parallelism": "single-gpu", "tokens": "uniform-random ids",
                "l2": "working set per step exceeds L2 (no flush)", "peaks": peaks["source"],
            },
            "clocks": {k: main_run["clocks"][k] for k in ("sm_mhz", "sm_max_mhz", "reasons")},
            # every step of the reference builds its ids and positions on the host (int64), copies them and
            # its decode metadata to the device, and reads the argmax back (reference:
            # src/scheduler/orca_scheduler.py:214-219, 250)
            "e2e": {"value": main_run["e2e_tok_s"], "unit": "tokens/s", "ms_per_step": main_run["e2e_ms_per_step"],
                    "h2d_bytes_per_step": 2 * args.batch * 8, "d2h_bytes_per_step": args.batch * 8},
            "gpu_launches": None,                                  # none of this repository's kernels run in this arm
            "roofline": {"bound": "hbm", "achieved": main_run["bytes_per_step"] / (main_run["ms"] / steps / 1e3) / 1e9,
                         "peak": peaks["hbm_gbs"], "unit": "GB/s"},
        }
        result["cuda_graphs"] = {key: value for key, value in model.cuda_graph_summary().items()
                                 if key in ("captured_graphs", "graph_replays", "capture_failures")}
        result["roofline"]["frac"] = result["roofline"]["achieved"] / result["roofline"]["peak"]
        if not args.small and not args.skip_prefill:
            result["prefill"] = measure_prefill(args.prefill_tokens)
        if not args.small and not args.skip_points:
            result["points"] = {"decode_b1": measure_decode(1, steps)["tok_s"],
                                "decode_b64": measure_decode(64, steps)["tok_s"]}
    return result


# ---------------------------------------------------------------------------------------------------------
# --design NAME: the design's prefill and decode throughput beside the closest other model of equal size, and
# its kernels alone.  Tefopel stands beside GPT-2; Gozunex (windowed attention over a cached latent, wkv layers,
# routed experts, several residual streams) beside Tefopel (windowed attention, wkv layers, a dense feed-forward);
# Zositar (chunked attention with normed heads and borrowed caches, routed experts with clamped activations and a
# gated dense feed-forward) beside a Tefopel of attention layers only; Pagatar (layers that norm their sublayers'
# results and end with an average over depth, a gated recurrence, latent attention without a window, attention with
# short convolutions, routed experts) beside a Gozunex of equal width, depth, heads, latent and experts; Suvunex (norms
# before and after each sublayer, attention beside gated linear attention, attention with mixed heads) beside a Tefopel in
# which every other layer is recurrent; Vozirax (state-space layers, differential attention, mixer and feed-forward side by
# side, experts without gates) beside a Suvunex of equal weights, whose kernels are the likes of most of its own.
DESIGN_SIZES = {"w1024": "w1024", "w2048": "w2048"}      # named sizes of config/tefopel.py and config/gozunex.py
DESIGN_CONTEXT = 2048


def design_arm(args):
    """Random models at sizes that resemble real layers: the design (three attention layers, then one wkv layer,
    repeated) and the closest other model with the same width, depth, heads, inner size per token and vocabulary:
    GPT-2 beside Tefopel, Tefopel beside Gozunex.  Per model: tokens/s of a 2,048-token prefill step (two prompts
    of 1,024) and of decode steps at batch 8 and 64 over 512-token prompts.  Then the design's kernels alone
    beside the like kernels of the other model, against the measured peaks."""
    import numpy as np
    import torch

    from pagedserve_b200.config.engine_config import EngineConfig
    from pagedserve_b200.config.gpt2 import GPT2Config
    from pagedserve_b200.engine.batch import StepEntry
    from pagedserve_b200.engine.engine import Engine
    from pagedserve_b200.kernels import microbench

    peaks = load_peaks()
    rng = np.random.default_rng(0)
    steps, warmup = min(args.steps, 64), max(args.warmup, 3)

    def configs(name):
        from pagedserve_b200.config import gozunex, pagatar, suvunex, tefopel, vozirax, zositar

        if args.design == "vozirax":
            # Suvunex of equal size: same width, depth and vocabulary, as many attention heads of the cached heads' size on as
            # many key heads, a recurrence in every other layer, and a dense feed-forward that makes the weights equal
            from pagedserve_b200.models import init_plan
            from pagedserve_b200.models.suvunex import build_suvunex_spec
            from pagedserve_b200.models.vozirax import build_vozirax_spec

            count = lambda spec: sum(math.prod(drawn[2] if len(drawn) > 2 else param.shape) for param, drawn in init_plan(spec))
            size = vozirax.NAMED_CONFIGS["vozirax-" + name]
            own = vozirax.named_config("vozirax-" + name)
            like = lambda ff: suvunex.repeating_config(
                width=size["width"], heads=size["heads"], head_dim=2 * size["head_dim"], kv_heads=size["kv_heads"],
                layers=size["layers"], vocab=size["vocab"], ff=ff, right_heads=size["width"] // 64, right_dim=64)
            spare = count(build_vozirax_spec(own)) - count(build_suvunex_spec(like(64)))
            ff = 64 + spare // (3 * size["width"] * size["layers"]) // 64 * 64
            return size, {"vozirax": own, "suvunex": like(ff)}
        if args.design == "suvunex":
            # Tefopel of equal size: same width, depth, heads and head size, a recurrent layer wherever the design has a
            # recurrence beside attention, windows that see every key, and a dense feed-forward that makes the weights equal
            size = suvunex.NAMED_CONFIGS["suvunex-" + name]
            like = tefopel.repeating_config(width=size["width"], heads=size["heads"], head_dim=size["head_dim"],
                                            ff=size["width"] * 35 // 8, layers=size["layers"],
                                            wkv_heads=size["width"] // 64, window=DESIGN_CONTEXT, vocab=size["vocab"], every=2)
            return size, {"suvunex": suvunex.named_config("suvunex-" + name), "tefopel": like}
        if args.design == "pagatar":
            # Gozunex of equal size: same width, depth, heads, flat and turning sizes, latent, experts and vocabulary;
            # its windows as long as the chunks, its recurrent layers where the gated recurrence stands, two residual
            # streams (one pass over the rows per sublayer, as the norm and sums behind a sublayer are here), no shared
            # expert
            size = pagatar.NAMED_CONFIGS["pagatar-" + name]
            like = gozunex.repeating_config(width=size["width"], heads=size["heads"], dim=size["head_dim"],
                                            rot_dim=size["rot_dim"], kv_rank=size["kv_rank"], experts=size["experts"],
                                            top=size["top"], ff=size["expert_ff"], layers=size["layers"],
                                            wkv_heads=size["width"] // 64, window=size["chunk"], vocab=size["vocab"])
            return size, {"pagatar": pagatar.named_config("pagatar-" + name), "gozunex": like}
        if args.design == "zositar":
            # Tefopel of equal size without wkv layers: same width, depth, heads and head size, a window as long as
            # the chunk, a dense feed-forward as wide as what one token uses of the experts
            size = zositar.NAMED_CONFIGS["zositar-" + name]
            like = tefopel.repeating_config(width=size["width"], heads=size["heads"], head_dim=size["head_dim"],
                                            ff=size["ff"], layers=size["layers"], wkv_heads=size["heads"],
                                            window=size["chunk"], vocab=size["vocab"], every=size["layers"] + 1)
            return size, {"zositar": zositar.named_config("zositar-" + name), "tefopel": like}
        if args.design == "gozunex":
            # Tefopel of equal size: same width, depth, heads, window and wkv heads; a head as wide as the cached
            # row's flat + turning parts; a dense feed-forward as wide as what one token uses of the experts
            size = gozunex.NAMED_CONFIGS["gozunex-" + name]
            like = tefopel.repeating_config(width=size["width"], heads=size["heads"], head_dim=size["dim"],
                                            ff=size["top"] * size["ff"] + (size.get("shared_ff") or 0),
                                            layers=size["layers"], wkv_heads=size["wkv_heads"], window=size["window"],
                                            vocab=size["vocab"])
            return size, {"gozunex": gozunex.named_config("gozunex-" + name), "tefopel": like}
        size = tefopel.NAMED_CONFIGS["tefopel-" + name]
        gpt2 = GPT2Config(n_layer=size["layers"], n_embd=size["width"], n_head=size["heads"], n_inner=size["ff"],
                          vocab_size=size["vocab"], n_positions=DESIGN_CONTEXT)
        return size, {"tefopel": tefopel.named_config("tefopel-" + name), "gpt2": gpt2}

    def timed(fn):
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        out = fn()
        end.record()
        torch.cuda.synchronize()
        return start.elapsed_time(end), out

    def measure(config):
        pages = 64 * (DESIGN_CONTEXT // 16) + 64
        engine = Engine.random(config, 0, EngineConfig(dtype=args.dtype, block_size=16, num_blocks=pages,
                                                       max_num_seqs=64, max_num_batched_tokens=2048,
                                                       max_model_len=DESIGN_CONTEXT))
        vocab = config.vocabulary_size
        result = {"weights_mb": engine.model.weight_bytes() / 1e6}
        # prefill: two prompts of 1,024 in one step; the shape is captured as a CUDA graph after a few sightings
        rehearsals = max(3, getattr(engine.runner, "MIXED_SHAPE_SIGHTINGS", 2) + 1)
        times = []
        for repeat in range(rehearsals + 5):
            entries = [StepEntry(1000 + i, rng.integers(0, vocab, 1024).tolist(), [1023]) for i in range(2)]
            ms, _ = timed(lambda: engine.step(entries))
            if repeat >= rehearsals:
                times.append(ms)
            for i in range(2):
                engine.finish(1000 + i)
        result["prefill_tok_s"] = 2048 / (statistics.median(times) / 1e3)
        result["prefill_ms"] = statistics.median(times)
        for batch in (8, 64):
            tokens = []
            for first in range(0, batch, 4):
                group = range(first, min(batch, first + 4))
                logits = engine.step([StepEntry(i, rng.integers(0, vocab, 512).tolist(), [511]) for i in group])
                tokens += logits.argmax(-1).tolist()
            entries = [StepEntry(i, [tokens[i]]) for i in range(batch)]
            warm = engine.decode(entries, [0.0] * batch, [0] * batch, steps=warmup)
            entries = [StepEntry(i, [int(warm[-1, i])]) for i in range(batch)]
            with ClockSampler() as clocks:
                ms, out = timed(lambda: engine.decode(entries, [0.0] * batch, [0] * batch, steps=steps))
            assert out.shape == (steps, batch)
            for i in range(batch):
                engine.finish(i)
            result[f"decode_b{batch}_tok_s"] = batch * steps / (ms / 1e3)
            result[f"decode_b{batch}_ms_per_step"] = ms / steps
            result[f"decode_b{batch}_clocks"] = clocks.summary()
        engine.check_status()
        del engine
        torch.cuda.empty_cache()
        return result

    report = {"impl": "ours", "design": args.design, "dtype": args.dtype, "data": "synthetic (random weights, uniform ids)",
              "steps": steps, "warmup": warmup, "peaks": peaks, "models": {}, "kernels": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
        size, pair = configs(DESIGN_SIZES[name])
        report["models"][name] = {"size": size, **{kind: measure(config) for kind, config in pair.items()}}
        both = report["models"][name]
        design, like = list(pair)
        both[f"{design}_over_{like}"] = {key: both[design][key] / both[like][key]
                                         for key in ("prefill_tok_s", "decode_b8_tok_s", "decode_b64_tok_s")}
    if args.dtype == "bfloat16" and not args.skip_points and args.design == "gozunex":
        from pagedserve_b200.config import gozunex

        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]
        for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
            size = gozunex.NAMED_CONFIGS["gozunex-" + name]
            H, d, r, R, width = size["heads"], size["dim"], size["rot_dim"], size["kv_rank"], size["width"]
            row = R + r
            # attention over the one-plane cache of rows [latent | turning key] beside Tefopel's keys and values
            like = microbench.time_decode_attention(64, 1024, H, H, d, window=1024, softcap=50.0, sink=True)
            split = microbench.time_decode_attention(64, 1024, H, 1, row, window=1024, planes=1)
            kernels[f"decode_attention_{name}"] = {"tefopel": {**like, "frac_hbm": like["gbs"] / hbm},
                                                   "gozunex_split_key": {**split, "frac_hbm": split["gbs"] / hbm}}
            if row <= 128:          # what the engine runs from 32 single tokens on: the heads as query rows
                own = microbench.time_shared_position_attention(64, 1024, H, row, window=1024)
                kernels[f"decode_attention_{name}"]["gozunex"] = {**own, "frac_hbm": own["gbs"] / hbm}
                few = microbench.time_decode_attention(8, 1024, H, 1, row, window=1024, planes=1)
                few_like = microbench.time_decode_attention(8, 1024, H, H, d, window=1024, softcap=50.0, sink=True)
                few_rows = microbench.time_shared_position_attention(8, 1024, H, row, window=1024)
                kernels[f"decode_attention_b8_{name}"] = {"tefopel": {**few_like, "frac_hbm": few_like["gbs"] / hbm},
                                                          "gozunex": {**few, "frac_hbm": few["gbs"] / hbm},
                                                          "gozunex_heads_as_rows": {**few_rows,
                                                                                    "frac_hbm": few_rows["gbs"] / hbm}}
            if row in (64, 128) and d in (64, 128):
                like = microbench.time_prefill_attention(2, 1024, H, H, d, window=1024, softcap=50.0, sink=True)
                own = microbench.time_prefill_attention(2, 1024, H, 1, row, window=1024, planes=1)
                kernels[f"prefill_attention_{name}"] = {"tefopel": {**like, "frac_tensor": like["tflops"] / tensor},
                                                        "gozunex": {**own, "frac_tensor": own["tflops"] / tensor}}
            like = microbench.time_cache_write(2048, H, H, d, rot_dims=(d // 4) * 2)
            own = microbench.time_latent_prepare(2048, H, d, r, R)
            kernels[f"cache_write_{name}"] = {"tefopel": {"us": like["us"], "gbs": like["gbs"], "frac_hbm": like["gbs"] / hbm},
                                              "gozunex": {**own, "frac_hbm": own["gbs"] / hbm}}
            for label, tokens in (("prefill_2048", 2048), ("decode_b64", 64)):
                run = microbench.time_hyper_step(tokens, width, 2)
                kernels[f"streams_{label}_{name}"] = {**run, "frac_hbm": run["gbs"] / hbm}
            run = microbench.time_experts(2048, width, size["experts"], size["top"], size["ff"])
            kernels[f"experts_2048_tokens_{name}"] = {**run, "frac_tensor": run["tflops"] / tensor,
                                                      "dense_frac_tensor": run["dense_tflops"] / tensor}
    elif args.dtype == "bfloat16" and not args.skip_points and args.design == "vozirax":
        from pagedserve_b200.config import vozirax

        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]

        def of_hbm(run):
            return {**run, "frac_hbm": run["gbs"] / hbm}

        def of_tensor(run):
            return {**run, "frac_tensor": run["tflops"] / tensor}

        for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
            size = vozirax.NAMED_CONFIGS["vozirax-" + name]
            H, G, d, width = size["heads"], size["kv_heads"], size["head_dim"], size["width"]
            slot, inner, channels = 2 * d, size["ssm_heads"] * size["ssm_dim"], size["ssm_heads"] * size["ssm_dim"] + 2 * size["ssm_state"]
            for label, items, each in (("prefill_2x1024", 2, 1024), ("decode_b64", 64, 1), ("decode_b8", 8, 1)):
                kernels[f"recurrence_{label}_{name}"] = {
                    "suvunex": of_hbm(microbench.time_gla(items, each, width // 64, 64, 64)),
                    "vozirax": of_hbm(microbench.time_ssd(items, each, size["ssm_heads"], 1, size["ssm_state"], size["ssm_dim"]))}
            # attention with two maps per head: twice the query heads on the same cache, results left as float32
            for batch in (8, 64):
                kernels[f"decode_attention_b{batch}_{name}"] = {
                    "suvunex": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, slot, sink=True, as_rows=True)),
                    "vozirax": of_hbm(microbench.time_decode_attention(batch, 1024, 2 * H, G, slot, as_rows=True, wide=True))}
            kernels[f"prefill_attention_{name}"] = {
                "suvunex": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, slot, sink=True)),
                "vozirax": of_tensor(microbench.time_prefill_attention(2, 1024, 2 * H, G, slot, wide=True))}
            for label, tokens in (("prefill_2048", 2048), ("decode_b64", 64), ("decode_b8", 8)):
                items = 2 if tokens > 64 else tokens
                kernels[f"cache_write_{label}_{name}"] = {
                    "suvunex": of_hbm(microbench.time_head_norm_cache_write(tokens, H, G, slot, rot_dims=slot)),
                    "vozirax": of_hbm(microbench.time_diff_prepare(tokens, H, G, d, 2 * d)),
                    "vozirax_combine": of_hbm(microbench.time_diff_combine(tokens, H, 2 * d, slot))}
                kernels[f"norms_{label}_{name}"] = {
                    "suvunex_close": of_hbm(microbench.time_sandwich_close(tokens, width)),
                    "tefopel_norm": of_hbm(microbench.time_layernorm(tokens, width)),
                    "vozirax_two_norms": of_hbm(microbench.time_norm_pair(tokens, width)),
                    "vozirax_gated_norm": of_hbm(microbench.time_group_norm(tokens, inner, 1))}
                kernels[f"convolution_{label}_{name}"] = {
                    "pagatar": of_hbm(microbench.time_short_conv(tokens, items, H, H, slot, 3)),
                    "suvunex": of_hbm(microbench.time_row_conv(tokens, items, width, 4)),
                    "vozirax": of_hbm(microbench.time_gated_conv(tokens, items, channels, 4, beside=inner))}
            like = microbench.time_experts(2048, width, size["experts"], size["top"], size["expert_ff"], score="sigmoid",
                                           normalize=False)
            own = microbench.time_experts(2048, width, size["experts"], size["top"], size["expert_ff"], score="sigmoid",
                                          form="relu_squared")
            kernels[f"experts_2048_tokens_{name}"] = {"pagatar": of_tensor(like), "vozirax": of_tensor(own)}
    elif args.dtype == "bfloat16" and not args.skip_points and args.design == "suvunex":
        from pagedserve_b200.config import suvunex

        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]

        def of_hbm(run):
            return {**run, "frac_hbm": run["gbs"] / hbm}

        def of_tensor(run):
            return {**run, "frac_tensor": run["tflops"] / tensor}

        for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
            size = suvunex.NAMED_CONFIGS["suvunex-" + name]
            H, d, width, G = size["heads"], size["head_dim"], size["width"], suvunex.repeating_config(**size).layers[0][
                "mixer"]["left"]["kv_heads"]
            # the two recurrences, each with the heads it has at this width
            for label, items, each in (("prefill_2x1024", 2, 1024), ("decode_b64", 64, 1), ("decode_b8", 8, 1)):
                kernels[f"recurrence_{label}_{name}"] = {
                    "tefopel": of_hbm(microbench.time_wkv(items, each, width // 64, 64, width)),
                    "suvunex": of_hbm(microbench.time_gla(items, each, size.get("right_heads", H), size.get("right_dim", d),
                                                          size.get("right_dim", d)))}
            if d > 64:                                       # larger heads than the other recurrence has
                for label, items, each in (("prefill_2x1024", 2, 1024), ("decode_b64", 64, 1)):
                    kernels[f"recurrence_{label}_{name}"]["suvunex_large_heads"] = of_hbm(microbench.time_gla(items, each, H, d, d))
            # attention whose heads are mixed, with the mixing kernel, and plain attention of equal heads
            for batch in (8, 64):
                kernels[f"decode_attention_b{batch}_{name}"] = {
                    "tefopel": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, d, softcap=50.0, sink=True)),
                    "suvunex_left": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, d, sink=True, as_rows=True)),
                    "suvunex_mixed": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, d, sink=True, mixed=True,
                                                                            as_rows=True))}
            kernels[f"prefill_attention_{name}"] = {
                "tefopel": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, softcap=50.0, sink=True)),
                "suvunex_left": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, sink=True)),
                "suvunex_mixed": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, sink=True, mixed=True))}
            for label, tokens in (("prefill_2048", 2048), ("decode_b64", 64), ("decode_b8", 8)):
                like = microbench.time_cache_write(tokens, H, G, d, rot_dims=(d // 4) * 2)
                kernels[f"cache_write_{label}_{name}"] = {
                    "tefopel": {"us": like["us"], "gbs": like["gbs"], "frac_hbm": like["gbs"] / hbm},
                    "suvunex": of_hbm(microbench.time_head_norm_cache_write(tokens, H, G, d, rot_dims=d))}
                # what stands between two sublayers: a norm there, the close of one and the opening of the next here
                kernels[f"between_sublayers_{label}_{name}"] = {
                    "tefopel_norm": of_hbm(microbench.time_layernorm(tokens, width)),
                    "pagatar_close": of_hbm(microbench.time_post_norm_add(tokens, width, 2, size["layers"] // 2 + 1)),
                    "suvunex_close": of_hbm(microbench.time_sandwich_close(tokens, width)),
                    "suvunex_convolution": of_hbm(microbench.time_row_conv(tokens, 2 if tokens > 64 else tokens, width, 4)),
                    "pagatar_convolution": of_hbm(microbench.time_short_conv(tokens, 2 if tokens > 64 else tokens, H, H, d, 3))}
    elif args.dtype == "bfloat16" and not args.skip_points and args.design == "pagatar":
        from pagedserve_b200.config import pagatar

        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]

        def of_hbm(run):
            return {**run, "frac_hbm": run["gbs"] / hbm}

        for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
            size = pagatar.NAMED_CONFIGS["pagatar-" + name]
            H, d, width, entries = size["heads"], size["head_dim"], size["width"], size["layers"] // 2 + 1
            # the gated recurrence beside the recurrence with a matrix state per head, at equal width
            for label, items, each in (("prefill_2x1024", 2, 1024), ("decode_b64", 64, 1), ("decode_b8", 8, 1)):
                kernels[f"recurrence_{label}_{name}"] = {
                    "gozunex": of_hbm(microbench.time_wkv(items, each, width // 64, 64, width)),
                    "pagatar": of_hbm(microbench.time_mingru(items, each, width))}
            # what closes a sublayer: the norm, the residual sum and the average over depth (a layer in the middle of
            # the model) beside the update of two residual streams
            for label, tokens in (("prefill_2048", 2048), ("decode_b64", 64)):
                kernels[f"sublayer_close_{label}_{name}"] = {
                    "gozunex": of_hbm(microbench.time_hyper_step(tokens, width, 2)),
                    "pagatar": of_hbm(microbench.time_post_norm_add(tokens, width, 2, entries))}
                # what stands between the projections and attention: the convolution over q | k | v beside the kernel
                # that turns queries and keys and fills the pages
                like = microbench.time_cache_write(tokens, H, H, d, rot_dims=(d // 4) * 2)
                kernels[f"after_projection_{label}_{name}"] = {
                    "tefopel": {"us": like["us"], "gbs": like["gbs"], "frac_hbm": like["gbs"] / hbm},
                    "pagatar_convolution": of_hbm(microbench.time_short_conv(tokens, 2 if tokens > 64 else tokens, H, H, d, 3)),
                    "pagatar_norm_turn_write": of_hbm(microbench.time_head_norm_cache_write(tokens, H, H, d, rot_dims=d))}
    elif args.dtype == "bfloat16" and not args.skip_points and args.design == "zositar":
        from pagedserve_b200.config import zositar

        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]

        def of_hbm(run):
            return {**run, "frac_hbm": run["gbs"] / hbm}

        def of_tensor(run):
            return {**run, "frac_tensor": run["tflops"] / tensor}

        for name in (args.design_sizes.split(",") if args.design_sizes else DESIGN_SIZES):
            size = zositar.NAMED_CONFIGS["zositar-" + name]
            H, G, d, width, chunk = size["heads"], size["kv_heads"], size["head_dim"], size["width"], size["chunk"]
            form = ("clamped_swish", 7.0, 7.0, zositar.EXPERT_SIGMOID_SLOPE)
            # the same attention kernels with a chunked mask beside a window of the chunk's length (with Tefopel's
            # score cap and sinks); whole chunks, and chunks that end inside the prompt
            for batch in (8, 64):
                kernels[f"decode_attention_b{batch}_{name}"] = {
                    "tefopel": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, d, window=chunk, softcap=50.0, sink=True)),
                    "zositar": of_hbm(microbench.time_decode_attention(batch, 1024, H, G, d, chunk=chunk))}
            kernels[f"decode_attention_b64_quarter_chunks_{name}"] = {
                "tefopel": of_hbm(microbench.time_decode_attention(64, 1024, H, G, d, window=chunk // 4, softcap=50.0, sink=True)),
                "zositar": of_hbm(microbench.time_decode_attention(64, 1024, H, G, d, chunk=chunk // 4))}
            if d in (64, 128):
                kernels[f"prefill_attention_{name}"] = {
                    "tefopel": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, window=chunk, softcap=50.0, sink=True)),
                    "zositar": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, chunk=chunk))}
                kernels[f"prefill_attention_quarter_chunks_{name}"] = {
                    "tefopel": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, window=chunk // 4, softcap=50.0, sink=True)),
                    "zositar": of_tensor(microbench.time_prefill_attention(2, 1024, H, G, d, chunk=chunk // 4))}
            for label, tokens in (("prefill_2048", 2048), ("decode_b64", 64)):
                like = microbench.time_cache_write(tokens, H, G, d, rot_dims=(d // 4) * 2)
                kernels[f"cache_write_{label}_{name}"] = {
                    "tefopel": {"us": like["us"], "gbs": like["gbs"], "frac_hbm": like["gbs"] / hbm},
                    "zositar": of_hbm(microbench.time_head_norm_cache_write(tokens, H, G, d, rot_dims=(d // 4) * 2))}
            like = microbench.time_experts(2048, width, size["experts"], size["top"], size["expert_ff"])
            own = microbench.time_experts(2048, width, size["experts"], size["top"], size["expert_ff"], score="sigmoid",
                                          normalize=False, form=form)
            kernels[f"experts_2048_tokens_{name}"] = {"gozunex": of_tensor(like), "zositar": of_tensor(own)}
    elif args.dtype == "bfloat16" and not args.skip_points:
        hbm, tensor = peaks["hbm_gbs"], peaks["bf16_tflops"]
        kernels = report["kernels"]
        for hd in (64, 128):
            plain = microbench.time_decode_attention(64, 1024, 16, 16, hd)
            full = microbench.time_decode_attention(64, 1024, 16, 16, hd, window=1024, softcap=50.0, sink=True)
            kernels[f"decode_attention_hd{hd}"] = {
                "gpt2": {**plain, "frac_hbm": plain["gbs"] / hbm}, "tefopel": {**full, "frac_hbm": full["gbs"] / hbm}}
            plain = microbench.time_prefill_attention(2, 1024, 16, 16, hd)
            full = microbench.time_prefill_attention(2, 1024, 16, 16, hd, window=1024, softcap=50.0, sink=True)
            kernels[f"prefill_attention_hd{hd}"] = {
                "gpt2": {**plain, "frac_tensor": plain["tflops"] / tensor},
                "tefopel": {**full, "frac_tensor": full["tflops"] / tensor}}
        write = microbench.time_cache_write(2048, 16, 16, 64)
        kernels["cache_write_2048_tokens"] = {**write, "frac_hbm": write["gbs"] / hbm,
                                              "plain_write_frac_hbm": write["plain_write_gbs"] / hbm}
        for label, items, each in (("prefill_2x1024", 2, 1024), ("decode_b64", 64, 1), ("decode_b8", 8, 1)):
            run = microbench.time_wkv(items, each, 16, 64, 1024)
            kernels[f"wkv_{label}"] = {**run, "frac_hbm": run["gbs"] / hbm}
    print(json.dumps(report))
    return 0


def main():
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=256)
    parser.add_argument("--warmup", type=int, default=3)
    parser.add_argument("--impl", default="ours", choices=("ours", "reference"))
    parser.add_argument("--model", default="gpt2-124m")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--prompt-len", type=int, default=512)
    parser.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    parser.add_argument("--layers", type=int, default=None, help="run fewer layers than the configuration has")
    parser.add_argument("--skip-points", action="store_true")
    parser.add_argument("--skip-prefill", action="store_true")
    parser.add_argument("--small", action="store_true", help="profiling aid: only the default decode measurement")
    parser.add_argument("--prefill-only", action="store_true", help="profiling aid: only the prefill measurement")
    parser.add_argument("--prefill-tokens", type=int, default=2048,
                        help="tokens of the prefill step, in prompts of 1,024 (1024: one single prompt)")
    parser.add_argument("--serving", type=int, default=0, metavar="REQUESTS",
                        help="instead of the decode measurement: this many requests (prompts U[64,1024), outputs "
                             "U[32,256]) through the scheduler, chunked prefill under a 2,048-token budget")
    parser.add_argument("--design", default=None, choices=("tefopel", "gozunex", "zositar", "pagatar", "suvunex", "vozirax"),
                        help="instead of the default workload: prefill and decode throughput of this design at a few "
                             "sizes beside GPT-2 of equal size, and its kernels alone against the measured peaks")
    parser.add_argument("--design-sizes", default=None, help="comma-separated names out of: " + ", ".join(DESIGN_SIZES))
    args = parser.parse_args()

    world = int(os.environ.get("WORLD_SIZE", "1"))
    if args.gpus > 1 or world > 1:
        if int(os.environ.get("RANK", "0")) == 0:
            print(json.dumps({"error": "pagedserve_b200 is a single-GPU engine: bench.py runs at --gpus 1 only",
                              "n_gpus": max(args.gpus, world)}))
        return 2
    if args.impl == "reference":
        return reference_arm(args)
    if args.design:
        return design_arm(args)

    import numpy as np
    import torch

    from pagedserve_b200.config.engine_config import EngineConfig
    from pagedserve_b200.config.gpt2 import GPT2Config, NAMED_CONFIGS
    from pagedserve_b200.engine.batch import StepEntry
    from pagedserve_b200.engine.engine import Engine

    steps, warmup = args.steps, max(args.warmup, 3)
    sizes = dict(NAMED_CONFIGS[args.model])
    full_layers = sizes["n_layer"]
    if args.layers:
        sizes["n_layer"] = args.layers
    config = GPT2Config(**sizes)
    context_len = config.n_positions
    if args.prompt_len + warmup + steps + 2 > context_len:
        steps = context_len - args.prompt_len - warmup - 2
    peaks = load_peaks()

    max_batch = max(64, args.batch)
    pages = max_batch * (context_len // 16) + 64
    engine = Engine.random(config, 0, EngineConfig(dtype=args.dtype, block_size=16, num_blocks=pages,
                                                   max_num_seqs=max_batch, max_num_batched_tokens=2048))
    rng = np.random.default_rng(0)
    width = 2 if args.dtype == "bfloat16" else 4
    kv_bytes_per_token = 2 * config.n_layer * config.n_embd * width
    tensors = engine.model.tensors
    weight_bytes = sum(t.numel() * t.element_size() for name, t in tensors.items() if name != "wpe.weight")

    def prefill(batch, prompt_len, first_id):
        prompts = [rng.integers(0, config.vocab_size, prompt_len).tolist() for _ in range(batch)]
        tokens = []
        per_step = max(1, 2048 // prompt_len)
        for start in range(0, batch, per_step):
            chunk = range(start, min(batch, start + per_step))
            logits = engine.step([StepEntry(first_id + i, prompts[i], [prompt_len - 1]) for i in chunk])
            tokens += logits.argmax(-1).tolist()
        return tokens

    def measure_decode(batch, k_steps):
        ids = list(range(batch))
        tokens = prefill(batch, args.prompt_len, 0)
        entries = [StepEntry(i, [tokens[i]]) for i in ids]
        warm = engine.decode(entries, [0.0] * batch, [0] * batch, steps=warmup)
        entries = [StepEntry(i, [int(warm[-1, i])]) for i in ids]
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        launches_before = engine.ops.launches
        with ClockSampler() as clocks:
            torch.cuda.synchronize()
            start.record()
            out = engine.decode(entries, [0.0] * batch, [0] * batch, steps=k_steps)
            end.record()
            torch.cuda.synchronize()
        ms = start.elapsed_time(end)
        graph = engine.runner._graphs.get((batch, "sample"))
        launches = (graph.kernels * k_steps) if graph else (engine.ops.launches - launches_before)
        mean_context = args.prompt_len + warmup + (k_steps + 1) / 2.0
        for i in ids:
            engine.finish(i)
        assert out.shape == (k_steps, batch)
        return {"ms": ms, "tok_s": batch * k_steps / (ms / 1e3), "launches": launches,
                "bytes_per_step": weight_bytes + batch * mean_context * kv_bytes_per_token,
                "clocks": clocks.summary()}

    def measure_e2e(batch, k_steps, repeats=3):
        """The same metric through the scheduler, one host round trip per step: the timed region of every step
        holds the upload of the step's inputs from pinned host memory and the read of its sampled tokens.
        Exactly k_steps are timed, ``repeats`` times over (fresh requests each time); the median is reported:
        one run alone moves by 10 % with the load of the host it happens to share."""
        import gc

        runs = []
        # requests whose prompts ran in an earlier step are that many tokens ahead: where the context has room,
        # everybody gets as many tokens more, so that nobody finishes inside the timed steps
        head_start = -(-batch * args.prompt_len // 2048) + 1
        spare = max(0, min(head_start, context_len - args.prompt_len - (warmup + k_steps + 2)))
        for _ in range(repeats):
            scheduler = engine.make_scheduler(strategy="orca", max_num_seqs=batch, max_num_batched_tokens=2048)
            for _ in range(batch):
                scheduler.add_token_request(rng.integers(0, config.vocab_size, args.prompt_len).tolist(),
                                            max_new_tokens=warmup + k_steps + 2 + spare)
            while scheduler.waiting:
                scheduler.step()                       # prefill (untimed)
            for _ in range(warmup):
                scheduler.step()
            gc.collect()
            gc.disable()
            try:
                torch.cuda.synchronize()
                began = time.perf_counter()
                produced = 0
                for _ in range(k_steps):
                    produced += len(scheduler.step())
                torch.cuda.synchronize()
                seconds = time.perf_counter() - began
            finally:
                gc.enable()
            h2d = engine.runner.h2d_bytes
            scheduler.run_until_complete()
            runs.append((produced / seconds, seconds * 1e3 / k_steps))
        runs.sort()
        value, ms = runs[len(runs) // 2]
        return {"value": value, "unit": "tokens/s", "h2d_bytes_per_step": h2d,
                "d2h_bytes_per_step": batch * 4, "ms_per_step": ms, "repeats": repeats,
                "ms_per_step_runs": [round(r[1], 4) for r in runs]}

    def measure_prefill(tokens_total=2048, repeats=5):
        prompt_len = min(1024, context_len)
        count = tokens_total // prompt_len
        times = []
        # the step shape is captured as a CUDA graph once it has come back a few times
        rehearsals = max(3, getattr(engine.runner, "MIXED_SHAPE_SIGHTINGS", 2) + 1)
        for repeat in range(repeats + rehearsals):
            prompts = [rng.integers(0, config.vocab_size, prompt_len).tolist() for _ in range(count)]
            entries = [StepEntry(1000 + i, prompts[i], [prompt_len - 1]) for i in range(count)]
            torch.cuda.synchronize()
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            engine.step(entries)
            end.record()
            torch.cuda.synchronize()
            if repeat >= rehearsals:
                times.append(start.elapsed_time(end))
            for i in range(count):
                engine.finish(1000 + i)
        ms = statistics.median(times)
        T = count * prompt_len
        H, I, L = config.n_embd, config.inner_dim, config.n_layer
        gemm = 2.0 * T * L * (3 * H * H + H * H + 2 * H * I) + 2.0 * count * H * config.vocab_size
        attention = L * count * 4.0 * H * (prompt_len * (prompt_len + 1) / 2.0)
        flops = gemm + attention
        peak = peaks["bf16_tflops"] * 1e12 if args.dtype == "bfloat16" else 75e12
        return {"value": T / (ms / 1e3), "tokens": T, "ms": ms, "frac": flops / (ms / 1e3) / peak,
                "gflop": flops / 1e9}

    def measure_serving(requests, max_seqs=64):
        """Continuous batching: every request is queued at time 0; a step holds the decode tokens of the running
        requests and prompt portions of waiting ones under the token budget.  The last of three passes is
        reported: the earlier ones meet most step shapes for the first few times (a shape that keeps coming
        back is captured as a CUDA graph, a step of about 5 ms)."""
        import gc

        for _ in range(3):
            scheduler = engine.make_scheduler(strategy="sarathi", max_num_seqs=max_seqs, max_num_batched_tokens=2048,
                                              prefill_chunk_size=512, max_prefills_per_step=4)
            prompt_tokens = 0
            for _ in range(requests):
                prompt_len = int(rng.integers(64, 1024))
                output_len = max(1, min(int(rng.integers(32, 257)), context_len - prompt_len))
                scheduler.add_token_request(rng.integers(0, config.vocab_size, prompt_len).tolist(),
                                            max_new_tokens=output_len)
                prompt_tokens += prompt_len
            step_ms, produced = [], 0
            gc.collect()
            gc.disable()                   # a collection of the oldest generation in mid-pass is one long step
            try:
                torch.cuda.synchronize()
                began = time.perf_counter()
                while scheduler.waiting or scheduler.active:
                    before = time.perf_counter()
                    produced += len(scheduler.step())
                    step_ms.append((time.perf_counter() - before) * 1e3)
                torch.cuda.synchronize()
                seconds = time.perf_counter() - began
            finally:
                gc.enable()
            engine.cache.check_invariants()
        step_ms.sort()
        return {"impl": "ours", "workload": "continuous batching", "model": args.model, "dtype": args.dtype,
                "requests": requests, "max_num_seqs": max_seqs, "max_num_batched_tokens": 2048,
                "prompt_tokens": prompt_tokens, "output_tokens": produced, "seconds": seconds,
                "output_tok_s": produced / seconds, "total_tok_s": (prompt_tokens + produced) / seconds,
                "steps": len(step_ms), "step_ms_median": step_ms[len(step_ms) // 2],
                "step_ms_p90": step_ms[int(len(step_ms) * 0.9)], "step_ms_max": step_ms[-1]}

    if args.prefill_only:
        print(json.dumps({"impl": "ours", "prefill": measure_prefill(args.prefill_tokens, repeats=3)}))
        return 0
    if args.serving:
        print(json.dumps(measure_serving(args.serving)))
        return 0
    main_run = measure_decode(args.batch, steps)
    e2e = measure_e2e(args.batch, steps)
    result = {
        "metric": "decode tok/s at batch 1/8/64; prefill tok/s at 2,048 tokens (GPT-2 124M)",
        "value": main_run["tok_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": main_run["ms"] / steps, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16" if args.dtype == "bfloat16" else "fp32", "data": "synthetic",
        "impl": "ours",
        "config": {
            "model": args.model, "weights": "random(seed 0)", "n_layer": config.n_layer,
            "n_layer_full": full_layers, "n_embd": config.n_embd, "n_head": config.n_head,
            "n_inner": config.inner_dim, "vocab_size": config.vocab_size, "n_positions": config.n_positions,
            "global_batch": args.batch, "seq_len": context_len, "prompt_len": args.prompt_len,
            "generated": steps, "block_size": 16, "parallelism": "single-gpu",
            "tokens": "uniform-random ids", "l2": "working set per step exceeds L2 (no flush)",
            "peaks": peaks["source"],
        },
        "clocks": {k: main_run["clocks"][k] for k in ("sm_mhz", "sm_max_mhz", "reasons")},
        "e2e": e2e,
        "gpu_launches": main_run["launches"],
        "roofline": {"bound": "hbm", "achieved": main_run["bytes_per_step"] / (main_run["ms"] / steps / 1e3) / 1e9,
                     "peak": peaks["hbm_gbs"], "unit": "GB/s"},
    }
    result["roofline"]["frac"] = result["roofline"]["achieved"] / result["roofline"]["peak"]
    if not args.small and not args.skip_prefill:
        result["prefill"] = measure_prefill(args.prefill_tokens)
    if not args.small and not args.skip_points:
        result["points"] = {"decode_b1": measure_decode(1, steps)["tok_s"],
                            "decode_b64": measure_decode(64, steps)["tok_s"]}
    print(json.dumps(result))
    return 0


if __name__ == "__main__":
    sys.exit(main())
