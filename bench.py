"""Throughput of the engine on one B200: decode and prefill at Qwen3-0.6B dimensions (the
default, the headline), and the serving workloads of the 8B and 32B dimensions.

``python bench.py --gpus 1 --steps K --warmup W`` prints ONE JSON line.  A step is one decode
step of a batch of 8 requests whose contexts start at 2,048 tokens (context limit 4,096), random
weights, bfloat16.

* ``value``: decoded tokens per second, device-timed with CUDA events over K replays of the
  decode step (the metadata of every step uploaded from pinned memory, no host synchronisation
  between steps).
* ``e2e``: the same through the public token-level API (``Engine.submit`` / ``Engine.step``),
  which every step uploads the step's inputs from pinned host memory and copies the sampled
  tokens back to pinned host memory (the engine plans up to 32 decode steps at once, keeps two
  launched ahead of the one it reads, and a call of ``step`` returns the tokens of one of them).
* ``prefill``: one prompt of 2,048 tokens through the step function.
* ``roofline``: bytes a decode step must read (every weight once + the cache of the live
  requests) / time / measured HBM bandwidth.
* ``points``: decode at batch 1 and 64; decode at batch 8 from a context of 16,384 tokens (with its
  fraction of the HBM roofline), a prefill of 8,192 tokens (with its fraction of the tensor peak) and
  decode of one request alone at a context of 32,768.

Every step reads more than the 126 MB of L2 (the weights alone are 1.19 GB), so the inputs are
larger than L2 and no flush is needed between timed steps.

``--workload 8b`` / ``--workload 32b`` run the request mixes of those sizes at full depth through
``Engine.step`` (64 requests with prompts of 128 to 4,096 tokens and 128 new tokens, half of them
sampled at temperature 0.8, 2,048 prompt tokens a step; 8 requests with prompts of 4,096 to
16,384 tokens and 256 new tokens) and print one JSON line with tokens per second, the time of a
decode step with every request live and its fraction of the HBM roofline.  ``--workload
arrivals`` replays 16 requests that arrive 20 ms apart at the 0.6B sizes (time to first token and
time per output token).

``--impl reference`` runs the unmodified reference installed under ``baseline/_ref`` on the same
decode workload through its own engine, or prints one line saying why it cannot.
"""

from __future__ import annotations

import argparse
import dataclasses
import json
import random
import statistics
import subprocess
import sys
import tempfile
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent

MODELS = {
    "0.6b": dict(vocab_size=151936, hidden_size=1024, intermediate_size=3072, num_hidden_layers=28,
                 num_attention_heads=16, num_key_value_heads=8, head_dim=128,
                 max_position_embeddings=40960, rope_theta=1_000_000.0, rms_norm_eps=1e-6,
                 tie_word_embeddings=True),
    "8b": dict(vocab_size=151936, hidden_size=4096, intermediate_size=12288, num_hidden_layers=36,
               num_attention_heads=32, num_key_value_heads=8, head_dim=128,
               max_position_embeddings=40960, rope_theta=1_000_000.0, rms_norm_eps=1e-6,
               tie_word_embeddings=False),
    "32b": dict(vocab_size=151936, hidden_size=5120, intermediate_size=25600, num_hidden_layers=64,
                num_attention_heads=64, num_key_value_heads=8, head_dim=128,
                max_position_embeddings=40960, rope_theta=1_000_000.0, rms_norm_eps=1e-6,
                tie_word_embeddings=False),
}
MODEL = MODELS["0.6b"]
CONTEXT_LIMIT = 4096
PROMPT_TOKENS = 2048
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}
METRIC = "decode tok/s @ batch 8 (Qwen3-0.6B dims, bf16, context from 2,048)"


def peaks() -> tuple[dict, str]:
    path = ROOT / "MEASURED_PEAKS.json"
    if path.is_file():
        try:
            data = json.loads(path.read_text())
            flat = {}

            def walk(node):
                if isinstance(node, dict):
                    for key, value in node.items():
                        if isinstance(value, (int, float)) and key in FALLBACK_PEAKS:
                            flat.setdefault(key, float(value))
                        else:
                            walk(value)
                elif isinstance(node, list):
                    for value in node:
                        walk(value)

            walk(data)
            if "hbm_gbs" in flat and "bf16_tflops" in flat:
                return {**FALLBACK_PEAKS, **flat}, "measured"
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    """nvidia-smi clocks and throttle reasons while the timed regions run."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self) -> None:
        self.process = None
        self.lines: list[str] = []
        self.spans: list[tuple[int, int]] = []

    def start(self) -> None:
        try:
            self.process = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "20"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.process = None

    def _read(self) -> None:
        for line in self.process.stdout:
            self.lines.append(line.strip())

    def mark(self) -> int:
        return len(self.lines)

    def span(self, first: int) -> None:
        """The samples from ``first`` to now were taken under a timed region."""
        self.spans.append((first, len(self.lines)))

    def stop(self) -> None:
        if self.process is not None:
            self.process.terminate()

    def summary(self) -> dict:
        sm, sm_max, reasons = [], 0, set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        chosen = [line for first, last in self.spans for line in self.lines[first:last]]
        for line in chosen or self.lines[-3:]:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) != 6:
                continue
            try:
                sm.append(int(parts[0]))
                sm_max = max(sm_max, int(parts[1]))
            except ValueError:
                continue
            for name, value in zip(names, parts[2:]):
                if value.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": int(statistics.median(sm)) if sm else None, "sm_max_mhz": sm_max or None,
                "reasons": sorted(reasons), "samples": len(sm)}


def random_prompt(rng: random.Random, count: int, vocab: int = MODEL["vocab_size"]) -> list[int]:
    return [rng.randrange(vocab) for _ in range(count)]


# --------------------------------------------------------------------------- the reference arm
def reference_arm(args) -> int:
    """The unmodified reference from ``baseline/_ref`` on the decode workload: the same model sizes
    with random weights, ``--batch`` prompts of 2,048 tokens prefilled untimed, then K decode steps
    through its own ``Engine.step`` (its scheduler, executor, CUDA kernels and decode graphs).
    Nothing of this repository's package is imported here.  If the reference cannot run on this
    machine, one line says why, in its own words."""
    import types

    line = {"impl": "reference", "metric": METRIC, "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": max(args.warmup, 3), "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic: uniform random token ids, random weights N(0, 0.02)"}
    warmup, steps, batch = max(args.warmup, 3), args.steps, args.batch
    stage = "import"
    try:
        sys.path.insert(0, str(ROOT / "baseline" / "_ref"))
        import torch
        from tinyvllm.engine import Engine
        from tinyvllm.executor import Executor
        from tinyvllm.models.qwen3 import Qwen3Config, Qwen3ForCausalLM
        from tinyvllm.request import SamplingParams
        from tinyvllm.scheduler import Scheduler

        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device is visible")
        stage = "model"
        layers = args.layers
        config = Qwen3Config.from_hf(types.SimpleNamespace(
            model_type="qwen3", hidden_act="silu", eos_token_id=None,
            **{**MODEL, "num_hidden_layers": layers}))
        with torch.inference_mode():
            model = Qwen3ForCausalLM(config, device="cuda", dtype=torch.bfloat16)
            generator = torch.Generator(device="cuda").manual_seed(0)
            for _, parameter in model.named_parameters():
                if parameter.dim() >= 2:
                    parameter.normal_(0.0, 0.02, generator=generator)
                else:
                    parameter.fill_(1.0)
            model.eval()
        stage = "engine (its CUDA kernels are built here)"
        new_tokens = steps + warmup + 64
        block = 16
        blocks = batch * (-(-(PROMPT_TOKENS + new_tokens + 64) // block)) + 256
        budget = max(4096, batch)
        executor = Executor(model, block_size=block, num_blocks=blocks, max_model_len=CONTEXT_LIMIT,
                            max_num_seqs=batch, attention_backend="cuda", enforce_eager=False)
        scheduler = Scheduler(max_active_requests=batch, max_step_requests=batch, max_scheduled_tokens=budget,
                              prefill_chunk_size=2048, max_model_len=CONTEXT_LIMIT, prefill_reserve_tokens=0,
                              prefill_reserve_requests=0, kv_block_size=block, kv_num_blocks=blocks,
                              eos_token_ids=None, enable_prefix_caching=False)
        engine = Engine(scheduler, executor)
        stage = "prefill"
        rng = random.Random(batch)
        sampling = SamplingParams(max_new_tokens=new_tokens, temperature=0.0, ignore_eos=True)
        ids = [engine.submit(random_prompt(rng, PROMPT_TOKENS), sampling) for _ in range(batch)]
        started = set()
        while len(started) < batch:                      # untimed: until every request has its first token
            for event in engine.step().token_events:
                started.add(event.request_id)
        stage = "decode"
        sampler = ClockSampler()
        sampler.start()
        for _ in range(warmup):
            engine.step()
        torch.cuda.synchronize()
        mark = sampler.mark()
        wall = time.perf_counter()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        tokens = 0
        for _ in range(steps):
            tokens += len(engine.step().token_events)
        end.record()
        torch.cuda.synchronize()
        elapsed_ms = max(start.elapsed_time(end), (time.perf_counter() - wall) * 1e3)
        sampler.span(mark)
        sampler.stop()
        if tokens != batch * steps:
            raise RuntimeError(f"{tokens} tokens came back from {steps} steps of {batch} requests")
        value = tokens / (elapsed_ms / 1e3)
        line.update({
            "value": round(value, 1), "ms_per_step": round(elapsed_ms / steps, 4),
            "config": {"model": "Qwen3-0.6B dims", "layers": layers, "layers_of_config": MODEL["num_hidden_layers"],
                       "global_batch": batch, "seq_len": CONTEXT_LIMIT, "prompt_tokens": PROMPT_TOKENS,
                       "kv_block_size": block, "attention_backend": "cuda", "cuda_graphs": True,
                       "parallelism": "single GPU", "timed": "Engine.step of the reference, host tokens in and out"},
            # the reference has no device-only loop: its one number is end to end
            "e2e": {"value": round(value, 1), "unit": "tokens/s", "h2d_bytes_per_step": None,
                    "d2h_bytes_per_step": batch * 8},
            "clocks": sampler.summary(),
        })
        for request_id in ids:
            engine.cancel(request_id)
    except ModuleNotFoundError as exc:
        line = {"impl": "reference",
                "unavailable": f"the reference is not installed under baseline/_ref ({exc})"}
    except Exception as exc:  # noqa: BLE001  (whatever the reference raises is the reason)
        reason = " ".join(f"{type(exc).__name__}: {exc}".split())
        line = {"impl": "reference",
                "unavailable": f"the reference's own code refused at stage '{stage}': {reason[:400]}"}
    print(json.dumps(line))
    return 0


# ------------------------------------------------------------------------------- this engine
def new_tokens_of(steps: int, warmup: int) -> int:
    """Tokens a request of the decode measurement may generate: the warm-up and the timed steps of
    either measurement, and room for the steps a run has launched ahead when it is cut off."""
    return steps + warmup + 64


def clear_engine(engine) -> None:
    """Cancel whatever the engine holds and let a run in flight end, so that every page is back."""
    scheduler = engine.scheduler
    for request_id in list(scheduler.waiting) + list(scheduler.prefilling) + list(scheduler.decoding):
        engine.cancel(request_id)
    while engine.in_run:                # the steps launched ahead are read; the run's pages go back
        engine.step()
    scheduler.take_finished()


def make_engine(folder: str, layers: int, max_num_seqs: int, dtype: str = "bfloat16", eager: bool = False,
                new_tokens: int = 512, prompt_tokens: int = PROMPT_TOKENS):
    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.models import Qwen3Config

    config = Qwen3Config(**{**MODEL, "num_hidden_layers": layers})
    Path(folder, "config.json").write_text(json.dumps(config.to_json()))
    kv_bytes_per_token = 2 * layers * MODEL["num_key_value_heads"] * MODEL["head_dim"] * 2
    context = max(CONTEXT_LIMIT, prompt_tokens + new_tokens + 16)     # more steps than the workload's 256 fit too
    kv_budget = kv_bytes_per_token * (max_num_seqs * (prompt_tokens + new_tokens + 64) + 8192 + 4096)
    engine_config = EngineConfig(
        model=folder, dtype=dtype, weights="random", seed=0, max_model_len=context,
        max_num_seqs=max_num_seqs, max_num_batched_tokens=max(4096, max_num_seqs),
        prefill_chunk_size=2048, prefill_reserve_tokens=0, prefill_reserve_requests=0,
        kv_block_size=16, kv_cache_memory_bytes=kv_budget,
        graph_batch_sizes=(max_num_seqs,), enforce_eager=eager)
    return Engine.from_config(engine_config)


def decode_bytes(engine, batch: int, mean_context: float) -> float:
    from tinyvllm_b200.engine.step import StepRunner

    weights = engine.runner.model.weight_bytes()
    per_token = StepRunner.bytes_per_token(engine.runner.model, engine.runner.dtype)
    return weights + batch * mean_context * per_token


LONG_CONTEXT = 16384           # context of the long-context decode point
LONG_PREFILL = 8192            # tokens of the long prefill point
LONE_CONTEXT = 32768           # context of the point with one request alone


def prefill_flops(layers: int, tokens: int) -> float:
    h, i, v = MODEL["hidden_size"], MODEL["intermediate_size"], MODEL["vocab_size"]
    nq, nkv, d = MODEL["num_attention_heads"], MODEL["num_key_value_heads"], MODEL["head_dim"]
    linear = layers * (h * (nq + 2 * nkv) * d + nq * d * h + h * 2 * i + i * h)
    attention = layers * 2 * nq * d * (tokens * (tokens + 1) / 2)     # QK^T and PV over the causal half
    return 2.0 * tokens * linear + 2.0 * attention + 2.0 * h * v


def run_decode(engine, batch: int, steps: int, warmup: int, sampler: ClockSampler | None,
               prompt_tokens: int = PROMPT_TOKENS):
    """Device-timed and end-to-end decode of ``batch`` requests; a dict of the figures."""
    import torch

    from tinyvllm_b200 import SamplingParams
    from tinyvllm_b200.engine.step import StepEntry
    from tinyvllm_b200.ops import kernels

    rng = random.Random(batch)
    sampling = SamplingParams(max_new_tokens=new_tokens_of(steps, warmup), ignore_eos=True)

    def fresh_batch():
        """``batch`` requests with their prompts in the cache, about to decode their second token."""
        clear_engine(engine)
        for _ in range(batch):
            engine.submit(random_prompt(rng, prompt_tokens), sampling)
        while engine.scheduler.prefilling or engine.scheduler.waiting:      # untimed prefill
            engine.step()
        assert len(engine.scheduler.decoding) == batch

    fresh_batch()

    # ---- end to end through the public API: submit/step with host tokens in and out
    for _ in range(warmup):
        engine.step()
    graph_steps_before = engine.graph_steps
    torch.cuda.synchronize()
    mark = sampler.mark() if sampler else 0
    start_wall = time.perf_counter()
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    e2e_steps = 0
    while e2e_steps < steps:            # a call of step() returns the tokens of the decode steps it read
        before = engine.graph_steps
        events = engine.step()
        ran = engine.graph_steps - before
        assert ran >= 1 and len(events.tokens) == batch * ran, "decode steps did not replay graphs"
        e2e_steps += ran
    end.record()
    torch.cuda.synchronize()
    e2e_ms = max(start.elapsed_time(end), (time.perf_counter() - start_wall) * 1e3)
    if sampler:
        sampler.span(mark)
    assert engine.graph_steps - graph_steps_before == e2e_steps
    bucket = engine.graphs.bucket_for(batch)
    h2d_bytes = bucket.host.numel() * 4
    d2h_bytes = batch * 4

    # ---- device-timed: K replays, inputs uploaded each step, no host synchronisation; a new batch,
    # so that both measurements walk the same contexts
    fresh_batch()
    scheduler = engine.scheduler
    plans = []
    for _ in range(warmup + steps):
        scheduled = scheduler.schedule()
        plans.append(scheduled)
        # commit with arbitrary tokens: only the bookkeeping advances, nothing is run here
        scheduler.commit(scheduled, {item.request_id: rng.randrange(MODEL["vocab_size"])
                                     for item in scheduled.items})

    def replay(scheduled):
        entries = [StepEntry(item.request_id, (rng.randrange(MODEL["vocab_size"]),), (0,))
                   for item in scheduled.items]
        params = [scheduler.requests[item.request_id].sampling for item in scheduled.items]
        engine.graphs.run(scheduled.cache_plan, entries, params, [0] * len(entries))

    contexts = []
    for scheduled in plans[:warmup]:
        replay(scheduled)
    torch.cuda.synchronize()
    launches_before = kernels.launch_count()
    mark = sampler.mark() if sampler else 0
    start.record()
    for scheduled in plans[warmup:]:
        contexts.append(statistics.mean(item.start + 1 for item in scheduled.items))
        replay(scheduled)
    end.record()
    torch.cuda.synchronize()
    if sampler:
        sampler.span(mark)
    device_ms = start.elapsed_time(end)
    assert kernels.launch_count() == launches_before      # everything ran from the graph
    kernels.check_finished_launches()
    clear_engine(engine)
    return {
        "tokens_per_s": batch * steps / (device_ms / 1e3), "ms_per_step": device_ms / steps,
        "e2e_tokens_per_s": batch * e2e_steps / (e2e_ms / 1e3), "h2d": h2d_bytes, "d2h": d2h_bytes,
        "launches_per_step": engine.graphs.launches_per_step(batch),
        "mean_context": statistics.mean(contexts),
    }


def run_prefill(engine, repeats: int = 5, tokens: int = PROMPT_TOKENS):
    import torch

    from tinyvllm_b200.engine.step import StepEntry

    rng = random.Random(99)
    runner = engine.runner
    times = []
    with torch.inference_mode():
        for index in range(repeats + 2):
            rid = f"prefill{tokens}-{index}"
            runner.open(rid)
            entry = StepEntry(rid, tuple(random_prompt(rng, tokens)), (tokens - 1,))
            torch.cuda.synchronize()
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            runner.run([entry])
            end.record()
            torch.cuda.synchronize()
            runner.close(rid)
            if index >= 2:
                times.append(start.elapsed_time(end))
    return statistics.median(times)


def eager_profile(args, warmup: int) -> int:
    """Decode steps and one prefill through the eager path, so that a profiler sees every kernel."""
    import torch

    from tinyvllm_b200 import SamplingParams

    rng = random.Random(0)
    with tempfile.TemporaryDirectory() as folder:
        engine = make_engine(folder, args.layers, args.batch, eager=True, new_tokens=new_tokens_of(args.steps, warmup))
        sampling = SamplingParams(max_new_tokens=warmup + args.steps + 4, ignore_eos=True)
        for _ in range(args.batch):
            engine.submit(random_prompt(rng, PROMPT_TOKENS), sampling)
        while engine.scheduler.prefilling or engine.scheduler.waiting:
            engine.step()
        torch.cuda.synchronize()
        for _ in range(warmup + args.steps):
            engine.step()
        torch.cuda.synchronize()
        clear_engine(engine)
        print("eager profile run: ok", run_prefill(engine, repeats=1), "ms prefill")
        engine.close()
    return 0


def headline(args, warmup: int) -> int:
    import gc

    import torch

    peak, peak_source = peaks()
    sampler = ClockSampler()
    sampler.start()
    with tempfile.TemporaryDirectory() as folder:
        engine = make_engine(folder, args.layers, max(args.batch, 1), new_tokens=new_tokens_of(args.steps, warmup))
        main_run = run_decode(engine, args.batch, args.steps, warmup, sampler)
        clocks = sampler.summary()
        prefill_ms = run_prefill(engine)
        weight_bytes = engine.runner.model.weight_bytes()
        bytes_step = decode_bytes(engine, args.batch, main_run["mean_context"])
        points = {}
        engine.close()
        del engine
        gc.collect()
        torch.cuda.empty_cache()
        if not args.no_points:
            for batch in (1, 64):
                with tempfile.TemporaryDirectory() as other:
                    point_engine = make_engine(other, args.layers, batch, new_tokens=new_tokens_of(args.steps, warmup))
                    result = run_decode(point_engine, batch, args.steps, warmup, None)
                    points[f"decode_b{batch}"] = round(result["tokens_per_s"], 1)
                    points[f"decode_b{batch}_e2e"] = round(result["e2e_tokens_per_s"], 1)
                    point_engine.close()
                    del point_engine
                    gc.collect()
                    torch.cuda.empty_cache()
            # further context lengths: decode at batch 8 from a context of 16,384 and a prefill of 8,192
            with tempfile.TemporaryDirectory() as other:
                long_steps = min(args.steps, 32)
                long_engine = make_engine(other, args.layers, 8, new_tokens=new_tokens_of(long_steps, warmup),
                                          prompt_tokens=LONG_CONTEXT)
                result = run_decode(long_engine, 8, long_steps, warmup, None, prompt_tokens=LONG_CONTEXT)
                long_bytes = decode_bytes(long_engine, 8, result["mean_context"])
                points["decode_b8_ctx16k"] = round(result["tokens_per_s"], 1)
                points["decode_b8_ctx16k_hbm_frac"] = round(
                    long_bytes / (result["ms_per_step"] / 1e3) / 1e9 / peak["hbm_gbs"], 4)
                long_ms = run_prefill(long_engine, repeats=3, tokens=LONG_PREFILL)
                points["prefill_8192"] = round(LONG_PREFILL / (long_ms / 1e3), 1)
                points["prefill_8192_frac"] = round(
                    prefill_flops(args.layers, LONG_PREFILL) / (long_ms / 1e3) / (peak["bf16_tflops"] * 1e12), 4)
                long_engine.close()
                del long_engine
                gc.collect()
                torch.cuda.empty_cache()
            # one request alone with a context of 32,768 (the decode attention cuts it over several
            # clusters a kv head, so that more than 64 of the SMs read its keys)
            with tempfile.TemporaryDirectory() as other:
                lone_steps = min(args.steps, 32)
                lone_engine = make_engine(other, args.layers, 1, new_tokens=new_tokens_of(lone_steps, warmup),
                                          prompt_tokens=LONE_CONTEXT)
                result = run_decode(lone_engine, 1, lone_steps, warmup, None, prompt_tokens=LONE_CONTEXT)
                lone_bytes = decode_bytes(lone_engine, 1, result["mean_context"])
                points["decode_b1_ctx32k"] = round(result["tokens_per_s"], 1)
                points["decode_b1_ctx32k_hbm_frac"] = round(
                    lone_bytes / (result["ms_per_step"] / 1e3) / 1e9 / peak["hbm_gbs"], 4)
                lone_engine.close()
                del lone_engine
                gc.collect()
                torch.cuda.empty_cache()
    sampler.stop()

    achieved_gbs = bytes_step / (main_run["ms_per_step"] / 1e3) / 1e9
    flops = prefill_flops(args.layers, PROMPT_TOKENS)
    line = {
        "metric": METRIC,
        "value": round(main_run["tokens_per_s"], 1),
        "unit": "tokens/s",
        "n_gpus": 1, "steps": args.steps, "warmup": warmup,
        "ms_per_step": round(main_run["ms_per_step"], 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: uniform random token ids, random weights N(0, 0.02)",
        "impl": "ours",
        "config": {
            "model": "Qwen3-0.6B dims", "layers": args.layers, "layers_of_config": MODEL["num_hidden_layers"],
            "hidden": MODEL["hidden_size"], "q_heads": MODEL["num_attention_heads"],
            "kv_heads": MODEL["num_key_value_heads"], "head_dim": MODEL["head_dim"],
            "intermediate": MODEL["intermediate_size"], "vocab": MODEL["vocab_size"],
            "tied": True, "global_batch": args.batch, "seq_len": CONTEXT_LIMIT,
            "prompt_tokens": PROMPT_TOKENS, "kv_block_size": 16, "parallelism": "single GPU",
            "l2": "inputs larger than L2 (weights 1.19 GB read every step)",
            "cuda_graphs": True, "peaks": peak_source,
        },
        "e2e": {"value": round(main_run["e2e_tokens_per_s"], 1), "unit": "tokens/s",
                "h2d_bytes_per_step": main_run["h2d"], "d2h_bytes_per_step": main_run["d2h"]},
        "gpu_launches": main_run["launches_per_step"] * args.steps,
        "prefill": {"value": round(PROMPT_TOKENS / (prefill_ms / 1e3), 1), "tokens": PROMPT_TOKENS,
                    "ms": round(prefill_ms, 3),
                    "frac": round(flops / (prefill_ms / 1e3) / (peak["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved_gbs, 1), "peak": peak["hbm_gbs"],
                     "unit": "GB/s", "frac": round(achieved_gbs / peak["hbm_gbs"], 4),
                     "bytes_per_step": int(bytes_step), "weight_bytes": int(weight_bytes)},
        "points": points,
        "clocks": clocks,
    }
    print(json.dumps(line))
    return 0


# ---------------------------------------------------------- serving workloads of the other sizes
SERVING = {
    # requests, shortest and longest prompt, new tokens, context limit, half of the requests sampled
    "8b": dict(requests=64, shortest=128, longest=4096, new_tokens=128, max_model_len=8192, sampled=True),
    "32b": dict(requests=8, shortest=4096, longest=16384, new_tokens=256, max_model_len=32768, sampled=False),
}


def serving_workload(args) -> int:
    """The request mix of the 8B or 32B sizes through ``Engine.step``: chunked prefill under 2,048
    prompt tokens a step beside the decodes, every request to its last token; one JSON line."""
    import torch

    from tinyvllm_b200 import EngineConfig, SamplingParams
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepRunner
    from tinyvllm_b200.models import Qwen3Config
    from tinyvllm_b200.ops import kernels

    which = args.workload
    work = SERVING[which]
    dims = dict(MODELS[which])
    layers_of_config = dims["num_hidden_layers"]
    if args.layers_given:
        dims["num_hidden_layers"] = args.layers
    layers = dims["num_hidden_layers"]
    peak, peak_source = peaks()
    requests, new = work["requests"], work["new_tokens"]
    with tempfile.TemporaryDirectory() as folder:
        Path(folder, "config.json").write_text(json.dumps(Qwen3Config(**dims).to_json()))
        kv_per_token = 2 * layers * dims["num_key_value_heads"] * dims["head_dim"] * 2
        sizes = tuple(s for s in (1, 2, 4, 8, 16, 32, 64) if s <= requests)
        config = EngineConfig(
            model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=work["max_model_len"],
            max_num_seqs=requests, max_num_batched_tokens=2048 + 64, prefill_chunk_size=2048,
            prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
            kv_cache_memory_bytes=kv_per_token * requests * (work["longest"] + new + 64),
            gpu_memory_utilization=0.95, graph_batch_sizes=sizes)
        began = time.perf_counter()
        engine = Engine.from_config(config)
        start_up_s = time.perf_counter() - began
        weight_bytes = engine.runner.model.weight_bytes()
        rng = random.Random(3)
        prompt_tokens = 0
        for index in range(requests):
            count = rng.randrange(work["shortest"], work["longest"] + 1)
            prompt_tokens += count
            if work["sampled"] and index % 2:
                sampling = SamplingParams(max_new_tokens=new, temperature=0.8, seed=index, ignore_eos=True)
            else:
                sampling = SamplingParams(max_new_tokens=new, ignore_eos=True)
            engine.submit(random_prompt(rng, count, dims["vocab_size"]), sampling)
        sampler = ClockSampler()
        sampler.start()
        torch.cuda.synchronize()
        mark = sampler.mark()
        began = time.perf_counter()
        done, first_token_s = {}, None
        full_ms, full_steps, full_context = 0.0, 0, []
        scheduler = engine.scheduler
        while engine.has_unfinished():
            all_decode = not scheduler.waiting and not scheduler.prefilling and len(scheduler.decoding) == requests
            if all_decode:
                # a decode step with every request live, timed by itself (the wait costs the run a
                # little of its overlap between host and device)
                torch.cuda.synchronize()
                context = sum(scheduler.requests[r].computed_tokens + 1 for r in scheduler.decoding)
                before, at = engine.steps_run, time.perf_counter()
            events = engine.step()
            if all_decode:
                torch.cuda.synchronize()
                ran = engine.steps_run - before
                if ran == 1:
                    full_ms += (time.perf_counter() - at) * 1e3
                    full_steps += 1
                    full_context.append(context)
            if first_token_s is None and events.tokens:
                first_token_s = time.perf_counter() - began
            for output in events.finished:
                done[output.request_id] = output
        torch.cuda.synchronize()
        seconds = time.perf_counter() - began
        sampler.span(mark)
        sampler.stop()
        kernels.check_finished_launches()
        assert len(done) == requests and all(len(o.output_token_ids) == new for o in done.values())
        engine.runner.manager.check()
        assert all(pool.free_count == pool.num_pages for pool in engine.runner.manager.pools)
        decode_ms = full_ms / full_steps if full_steps else None
        hbm = None
        if decode_ms:
            per_token = StepRunner.bytes_per_token(engine.runner.model, engine.runner.dtype)
            bytes_step = weight_bytes + statistics.mean(full_context) * per_token
            achieved = bytes_step / (decode_ms / 1e3) / 1e9
            hbm = {"bound": "hbm", "achieved": round(achieved, 1), "peak": peak["hbm_gbs"], "unit": "GB/s",
                   "frac": round(achieved / peak["hbm_gbs"], 4), "bytes_per_step": int(bytes_step)}
        line = {
            "metric": f"serving workload, Qwen3-{which.upper()} dims, bf16: new tokens/s over the whole run",
            "value": round(requests * new / seconds, 1), "unit": "tokens/s", "n_gpus": 1,
            "higher_is_better": True, "dtype": "bf16", "impl": "ours",
            "data": "synthetic: uniform random token ids, random weights N(0, 0.02)",
            "seconds": round(seconds, 3), "prompt_tokens_per_s": round(prompt_tokens / seconds, 1),
            "first_token_s": round(first_token_s or 0.0, 3),
            "decode_ms_per_step": round(decode_ms, 3) if decode_ms else None,
            "decode_tokens_per_s": round(requests / decode_ms * 1e3, 1) if decode_ms else None,
            "roofline": hbm,
            "config": {"model": f"Qwen3-{which.upper()} dims", "layers": layers, "layers_of_config": layers_of_config,
                       "requests": requests, "prompt_tokens": prompt_tokens, "new_tokens": new,
                       "shortest_prompt": work["shortest"], "longest_prompt": work["longest"],
                       "seq_len": work["max_model_len"], "prefill_tokens_per_step": 2048,
                       "half_sampled_at_0.8": work["sampled"], "kv_block_size": 16, "peaks": peak_source,
                       "weight_gb": round(weight_bytes / 1e9, 2), "start_up_s": round(start_up_s, 1)},
            "steps": engine.steps_run, "graph_steps": engine.graph_steps,
            "device_gb_peak": round(torch.cuda.max_memory_allocated() / 1e9, 1),
            "clocks": sampler.summary(),
        }
        engine.close()
    print(json.dumps(line))
    return 0


# ------------------------------------------- Gumapel beside a windowed Qwen3 of equal layer sizes
GUMAPEL_SIZES = {
    # width, q heads, kv heads, head size, feed-forward width (the layers of the 0.6B, 8B and 32B sizes)
    "0.6b": (1024, 16, 8, 128, 3072),
    "8b": (4096, 32, 8, 128, 12288),
    "32b": (5120, 64, 8, 128, 25600),
}
GUMAPEL_WINDOW, GUMAPEL_KEPT = 1024, 4
# (kernel of the new design, its counterpart in the windowed Qwen3) by what they do
LIKE_KERNELS = (
    ("stream_norm", "rms_norm", "pre-norm + residual sum"),
    ("qkv_prepare", "qk_norm_rope_store", "q/k norm or rotation + cache write"),
    ("attention_tiles", "attention_prefill_tc", "prompt attention"),
    ("attention_tiles_singles", "attention_decode", "decode attention"),
    ("gated_act", "silu_mul", "act(gate) * up"),
)


class KernelClock:
    """Times every call of the named functions of ``ops.kernels`` with CUDA events (the calls of one
    eager step); ``totals()`` gives name -> (calls, milliseconds) after a synchronize."""

    def __init__(self, names):
        from tinyvllm_b200.ops import kernels
        self.kernels, self.names, self.originals, self.marks = kernels, names, {}, []

    def __enter__(self):
        import torch
        for name in self.names:
            original = getattr(self.kernels, name)
            self.originals[name] = original

            def timed(*args, _original=original, _name=name, **kwargs):
                start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                start.record()
                result = _original(*args, **kwargs)
                end.record()
                self.marks.append((_name, start, end))
                return result
            setattr(self.kernels, name, timed)
        return self

    def __exit__(self, *exc):
        for name, original in self.originals.items():
            setattr(self.kernels, name, original)

    def totals(self):
        import torch
        torch.cuda.synchronize()
        out = {}
        for name, start, end in self.marks:
            calls, ms = out.get(name, (0, 0.0))
            out[name] = (calls + 1, ms + start.elapsed_time(end))
        return out


def gumapel_config(size: str, layers: int):
    from tinyvllm_b200.models import GumapelConfig
    from tinyvllm_b200.models.gumapel import GumapelLayer

    width, heads, kv, dim, ff = GUMAPEL_SIZES[size]
    made = []
    for index in range(layers):
        if index % 4 == 3:
            made.append(GumapelLayer(type="attention", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                                     window=GUMAPEL_WINDOW, v_mix=True, ff=ff))
        else:
            made.append(GumapelLayer(type="attention_2", heads=heads, kv_heads=kv, dim=dim, vdim=dim,
                                     scale=dim ** -0.5, window=GUMAPEL_WINDOW, keep_first=GUMAPEL_KEPT, rot_dims=dim,
                                     rot_base=500000.0, v_mix=True, ff=ff))
    return GumapelConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, layers=tuple(made))


def windowed_qwen3_config(size: str, layers: int):
    from tinyvllm_b200.models import Qwen3Config

    width, heads, kv, dim, ff = GUMAPEL_SIZES[size]
    return Qwen3Config(**{**MODELS["0.6b"], "hidden_size": width, "num_attention_heads": heads,
                          "num_key_value_heads": kv, "head_dim": dim, "intermediate_size": ff,
                          "num_hidden_layers": layers, "tie_word_embeddings": False,
                          "layer_windows": (GUMAPEL_WINDOW,) * layers})


def kernel_roofline(name: str, size: str, tokens: int, context: int, peak: dict) -> tuple[float, str]:
    """Microseconds the kernel ``name`` needs at the measured peaks for one layer of ``size``: ``tokens``
    new tokens whose requests hold ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = GUMAPEL_SIZES[size]
    seen = min(GUMAPEL_WINDOW, context)
    bytes_, flops = 0.0, 0.0
    if name == "stream_norm":
        bytes_ = tokens * width * (4 + 4 + 4 + 2)
    elif name == "rms_norm":
        bytes_ = tokens * width * 2 * 4
    elif name in ("qkv_prepare", "qk_norm_rope_store"):
        bytes_ = tokens * dim * 2 * ((heads + 2 * kv) + heads + 2 * kv)
    elif name in ("gated_act", "silu_mul"):
        bytes_ = tokens * ff * 2 * 3
    elif name in ("attention_tiles", "attention_prefill_tc", "attention_prefill"):
        pairs = sum(min(p + 1, GUMAPEL_WINDOW) for p in range(tokens))       # (query, key) pairs seen
        flops = 2.0 * heads * 2 * dim * pairs
    elif name in ("attention_tiles_singles", "attention_decode"):
        bytes_ = tokens * kv * seen * 2 * dim * 2
    if flops:
        return flops / (peak["bf16_tflops"] * 1e12) * 1e6, "tensor"
    return bytes_ / (peak["hbm_gbs"] * 1e9) * 1e6, "memory"


def gumapel_workload(args) -> int:
    """Prefill and decode of Gumapel at the layer sizes of the 0.6B, 8B and 32B models (random
    weights, ``--layers`` layers, default 4, window 1,024) beside a Qwen3 of the same sizes whose
    layers all have that window: tokens/s through the engine, and every kernel of the new design
    beside its counterpart with the fraction of its roofline.  One JSON line."""
    import torch

    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepEntry

    layers = args.layers if args.layers_given else 4
    batch, prompt, steps, warmup = args.batch, PROMPT_TOKENS, min(args.steps, 64), max(args.warmup, 3)
    peak, peak_source = peaks()
    names = sorted({n for pair in LIKE_KERNELS for n in pair[:2]} | {"attention_prefill", "attention_rows"})
    results = []
    sampler = ClockSampler()
    sampler.start()
    for size in GUMAPEL_SIZES:
        row = {"size": size}
        for label, config in (("gumapel", gumapel_config(size, layers)), ("qwen3_windowed", windowed_qwen3_config(size, layers))):
            with tempfile.TemporaryDirectory() as folder:
                Path(folder, "config.json").write_text(json.dumps(config.to_json()))
                engine = Engine.from_config(EngineConfig(
                    model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=CONTEXT_LIMIT,
                    max_num_seqs=batch, max_num_batched_tokens=4096, prefill_chunk_size=2048,
                    prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
                    kv_cache_memory_bytes=2 * 1024**3, graph_batch_sizes=(batch,)))
                decode = run_decode(engine, batch, steps, warmup, sampler, prompt_tokens=prompt)
                prefill_ms = run_prefill(engine, repeats=5, tokens=prompt)
                # one eager prompt step and one eager decode step, kernel by kernel
                runner = engine.runner
                rng = random.Random(5)
                with torch.inference_mode():
                    for r in range(batch):
                        runner.open(f"k{r}")
                    prompts = [StepEntry(f"k{r}", tuple(random_prompt(rng, prompt)), ()) for r in range(batch)]
                    def eager_step(entries):
                        plan = runner.plan(entries)
                        runner.execute(runner.build_context(entries, plan))
                        runner.manager.commit(plan)

                    # the GPU is kept busy (a spin kernel of a few milliseconds) while the host queues the
                    # step's launches behind it: the events then bracket device time, not the host's pace
                    for entry in prompts[1:]:
                        eager_step([entry])
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(20_000_000)
                        eager_step([prompts[0]])
                    by_prompt = clock.totals()
                    singles = [StepEntry(f"k{r}", (1,), (0,)) for r in range(batch)]
                    eager_step(singles)
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(20_000_000)
                        eager_step(singles)
                    by_decode = clock.totals()
                    for r in range(batch):
                        runner.close(f"k{r}")
                kernels_out = {}
                for phase, found, tokens in (("prefill", by_prompt, prompt), ("decode", by_decode, batch)):
                    for name, (calls, ms) in sorted(found.items()):
                        per_layer = 1e3 * ms / max(1, calls)
                        ideal, bound = kernel_roofline(name, size, tokens, prompt, peak)
                        kernels_out[f"{phase}:{name}"] = {
                            "calls": calls, "us_per_call": round(per_layer, 2), "roofline_us": round(ideal, 2),
                            "bound": bound, "frac": round(ideal / per_layer, 3) if per_layer > 0 else None}
                row[label] = {
                    "decode_tokens_per_s": round(decode["tokens_per_s"], 1), "decode_ms_per_step": round(decode["ms_per_step"], 4),
                    "prefill_tokens_per_s": round(prompt / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                    "weight_bytes": engine.runner.model.weight_bytes(), "kernels": kernels_out}
                engine.close()
                del engine
                torch.cuda.empty_cache()
        results.append(row)
    sampler.stop()
    print(json.dumps({
        "metric": "Gumapel beside a windowed Qwen3 of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "window": GUMAPEL_WINDOW, "kept_first": GUMAPEL_KEPT, "batch": batch,
                   "vocab": MODEL["vocab_size"], "sizes": {k: list(v) for k, v in GUMAPEL_SIZES.items()},
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"], "source": peak_source},
        "clocks": sampler.summary(), "results": results}))
    return 0


# ------------------------------------------------------------- Kelasun beside the dense Qwen3
KELASUN_SIZES = {
    # width, q heads, kv heads, head size, active feed-forward width (the layers of the 0.6B, 8B and 32B
    # sizes); latent layers: heads of head/2 plain + 64 rotated dimensions, latents as below
    "0.6b": (1024, 16, 8, 128, 3072),
    "8b": (4096, 32, 8, 128, 12288),
    "32b": (5120, 64, 8, 128, 25600),
}
KELASUN_LATENTS = {"0.6b": (384, 192), "8b": (1536, 256), "32b": (1536, 256)}     # q_rank, kv_rank
KELASUN_ROT, KELASUN_EXPERTS, KELASUN_TOP = 64, 8, 2
KELASUN_LIKE = (
    ("post_layer_norm", "rms_norm", "norm + residual sum"),
    ("projection_norm", "qk_norm_rope_store", "q/k norm (+ temperature; the dense model also rotates and stores)"),
    ("qkv_prepare", "qk_norm_rope_store", "cache write"),
    ("latent_prepare", "qk_norm_rope_store", "latent norms, rotation, cache write"),
    ("rotate_heads", "qk_norm_rope_store", "rotation of the queries' rotated part"),
    ("head_product", None, "up-projections a head (folded into q, applied to the attended latent)"),
    ("attention_tiles", "attention_prefill_tc", "prompt attention"),
    ("attention_tiles_singles", "attention_decode", "decode attention"),
    ("route_act", "silu_mul", "routing + activation"),
)


def kelasun_expert_width(ff: int) -> int:
    """A third of the dense feed-forward width, rounded down to a multiple of 64."""
    return ff // (KELASUN_TOP + 1) // 64 * 64


def kelasun_config(size: str, layers: int):
    from tinyvllm_b200.models import KelasunConfig
    from tinyvllm_b200.models.kelasun import KelasunExperts, KelasunLayer

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    q_rank, kv_rank = KELASUN_LATENTS[size]
    unit = kelasun_expert_width(ff)           # the chosen experts and the shared one together are as wide as the dense ff
    experts = KelasunExperts(KELASUN_EXPERTS, KELASUN_TOP, unit, ff - KELASUN_TOP * unit)
    made = []
    for index in range(layers):
        if index % 2 == 0:
            made.append(KelasunLayer(type="attention", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                                     q_temp=(0.4, 512), mlp=experts))
        else:
            made.append(KelasunLayer(type="latent_attention", heads=heads, dim=dim // 2, vdim=dim, scale=dim ** -0.5,
                                     q_rank=q_rank, kv_rank=kv_rank, rot_dim=KELASUN_ROT, rot_base=1000000.0,
                                     rot_scaling=(8.0, 4096.0, 32.0, 1.0), mlp=experts))
    return KelasunConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, postln_alpha=2.0, logit_scale=1.0,
                         layers=tuple(made))


def dense_qwen3_config(size: str, layers: int):
    from tinyvllm_b200.models import Qwen3Config

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    return Qwen3Config(**{**MODELS["0.6b"], "hidden_size": width, "num_attention_heads": heads,
                          "num_key_value_heads": kv, "head_dim": dim, "intermediate_size": ff,
                          "num_hidden_layers": layers, "tie_word_embeddings": False})


def kelasun_roofline(name: str, kind: str, size: str, tokens: int, context: int, peak: dict):
    """(microseconds at the measured peaks, what bounds it) of one call of kernel ``name`` in a layer of
    ``kind`` ("attention", "latent", "dense": the Qwen3 layer): ``tokens`` new tokens whose requests hold
    ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    q_rank, kv_rank = KELASUN_LATENTS[size]
    row, rot = kv_rank + KELASUN_ROT, KELASUN_ROT
    unit = kelasun_expert_width(ff)
    columns = KELASUN_EXPERTS * unit + (ff - KELASUN_TOP * unit)
    pairs = tokens * (tokens + 1) // 2 if context == tokens else tokens * context
    bytes_, flops = 0.0, 0.0
    if name == "post_layer_norm":
        bytes_ = tokens * width * (4 + 4 + 4 + 2)
    elif name == "rms_norm":
        bytes_ = tokens * width * 2 * 4
    elif name == "projection_norm":
        bytes_ = tokens * (heads + kv) * dim * 2 * 2
    elif name in ("qkv_prepare", "qk_norm_rope_store"):
        bytes_ = tokens * dim * 2 * ((heads + 2 * kv) + heads + 2 * kv) if name == "qk_norm_rope_store" \
            else tokens * dim * 2 * 2 * 2 * kv
    elif name == "latent_prepare":
        bytes_ = tokens * (q_rank + row) * 2 * 2
    elif name == "rotate_heads":
        bytes_ = tokens * heads * rot * 2 * 2
    elif name == "head_product":
        flops = 2.0 * tokens * heads * kv_rank * (dim // 2 + dim) / 2      # the two products of a layer, averaged
    elif name in ("route_act",):
        bytes_ = tokens * columns * 2 * 2
    elif name == "silu_mul":
        bytes_ = tokens * ff * 2 * 3
    elif name in ("attention_tiles", "attention_prefill_tc", "attention_prefill"):
        flops = 2.0 * heads * ((row + kv_rank) if kind == "latent" else 2 * dim) * pairs
    elif name in ("attention_tiles_singles", "attention_decode"):
        bytes_ = tokens * context * 2 * (row if kind == "latent" else kv * 2 * dim)
    if flops:
        return flops / (peak["bf16_tflops"] * 1e12) * 1e6, "tensor"
    return bytes_ / (peak["hbm_gbs"] * 1e9) * 1e6, "memory"


def kelasun_workload(args) -> int:
    """Prefill and decode of Kelasun at the layer sizes of the 0.6B, 8B and 32B models (random weights,
    ``--layers`` layers, default 4, attention and latent layers in turn, 8 experts of which 2 are used
    plus a shared one, together as wide as the dense feed-forward) beside a dense Qwen3 of the same
    sizes: tokens/s through the engine, and every kernel of the new design beside its counterpart with
    the fraction of its roofline.  One JSON line."""
    import torch

    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepEntry

    layers = args.layers if args.layers_given else 4
    batch, prompt, steps, warmup = args.batch, PROMPT_TOKENS, min(args.steps, 64), max(args.warmup, 3)
    peak, peak_source = peaks()
    names = sorted({n for pair in KELASUN_LIKE for n in pair[:2] if n} | {"attention_prefill", "attention_rows"})
    both_kinds = ("attention_tiles", "attention_tiles_singles", "attention_rows")
    results = []
    sampler = ClockSampler()
    sampler.start()
    sizes = [size for size in KELASUN_SIZES if not args.sizes or size in args.sizes.split(",")]
    for size in sizes:
        row = {"size": size}
        for label, config in (("kelasun", kelasun_config(size, layers)), ("qwen3_dense", dense_qwen3_config(size, layers))):
            with tempfile.TemporaryDirectory() as folder:
                Path(folder, "config.json").write_text(json.dumps(config.to_json()))
                engine = Engine.from_config(EngineConfig(
                    model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=CONTEXT_LIMIT,
                    max_num_seqs=batch, max_num_batched_tokens=4096, prefill_chunk_size=2048,
                    prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
                    kv_cache_memory_bytes=2 * 1024**3, graph_batch_sizes=(batch,)))
                decode = run_decode(engine, batch, steps, warmup, sampler, prompt_tokens=prompt)
                prefill_ms = run_prefill(engine, repeats=5, tokens=prompt)
                runner = engine.runner
                rng = random.Random(5)
                with torch.inference_mode():
                    for r in range(batch):
                        runner.open(f"k{r}")
                    prompts = [StepEntry(f"k{r}", tuple(random_prompt(rng, prompt)), ()) for r in range(batch)]

                    def eager_step(entries):
                        plan = runner.plan(entries)
                        runner.execute(runner.build_context(entries, plan))
                        runner.manager.commit(plan)

                    # the GPU is kept busy (a spin kernel) while the host queues the step's launches behind it:
                    # the events then bracket device time, not the host's pace
                    for entry in prompts[1:]:
                        eager_step([entry])
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step([prompts[0]])
                    torch.cuda.synchronize()
                    by_prompt = list(clock.marks)
                    singles = [StepEntry(f"k{r}", (1,), (0,)) for r in range(batch)]
                    eager_step(singles)
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step(singles)
                    torch.cuda.synchronize()
                    by_decode = list(clock.marks)
                    for r in range(batch):
                        runner.close(f"k{r}")
                kernels_out = {}
                for phase, marks, tokens in (("prefill", by_prompt, prompt), ("decode", by_decode, batch)):
                    found, seen = {}, {}
                    for name, start, end in marks:
                        kind = "dense"
                        if label == "kelasun":
                            # the two kinds of layers call the attention kernels in turn, the attention layer first
                            index = seen.get(name, 0)
                            seen[name] = index + 1
                            kind = ("attention", "latent")[index % 2] if name in both_kinds else \
                                "latent" if name in ("latent_prepare", "rotate_heads", "head_product") else "attention"
                        key = name if kind == "dense" or name not in both_kinds else f"{name}[{kind}]"
                        calls, ms, _ = found.get(key, (0, 0.0, kind))
                        found[key] = (calls + 1, ms + start.elapsed_time(end), kind)
                    for key, (calls, ms, kind) in sorted(found.items()):
                        per_call = 1e3 * ms / max(1, calls)
                        ideal, bound = kelasun_roofline(key.split("[")[0], kind, size, tokens, prompt, peak)
                        kernels_out[f"{phase}:{key}"] = {
                            "calls": calls, "us_per_call": round(per_call, 2), "roofline_us": round(ideal, 2),
                            "bound": bound, "frac": round(ideal / per_call, 3) if per_call > 0 else None}
                row[label] = {
                    "decode_tokens_per_s": round(decode["tokens_per_s"], 1), "decode_ms_per_step": round(decode["ms_per_step"], 4),
                    "prefill_tokens_per_s": round(prompt / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                    "weight_bytes": engine.runner.model.weight_bytes(), "kernels": kernels_out}
                engine.close()
                del engine
                torch.cuda.empty_cache()
        results.append(row)
    sampler.stop()
    print(json.dumps({
        "metric": "Kelasun beside a dense Qwen3 of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "batch": batch, "vocab": MODEL["vocab_size"],
                   "sizes": {k: list(v) for k, v in KELASUN_SIZES.items() if k in sizes},
                   "latents": {k: list(v) for k, v in KELASUN_LATENTS.items() if k in sizes}, "rot_dim": KELASUN_ROT,
                   "experts": KELASUN_EXPERTS, "top": KELASUN_TOP,
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"], "source": peak_source},
        "clocks": sampler.summary(), "results": results}))
    return 0


# ------------------------------------------- Bimolix beside Kelasun at equal layer sizes
BIMOLIX_CHUNK, BIMOLIX_TABLE_ROWS = 1024, 32
# FP32 multiply-adds outside the tensor cores: 148 SMs x 128 lanes x 2 flops at the 1,965 MHz the boards
# allow (a nominal figure; the recurrence is float32 by the design's rule, so its kernel cannot use bf16 tiles)
FP32_TFLOPS_NOMINAL = 148 * 128 * 2 * 1.965e9 / 1e12
# (kernel of the new design, its counterpart in Kelasun) by what they do
BIMOLIX_LIKE = (
    ("stream_norm", "post_layer_norm", "norm + residual sum"),
    ("qkv_prepare", "projection_norm + qkv_prepare", "q/k bias and norm, cache write"),
    ("attention_tiles", "attention_tiles[attention]", "prompt attention"),
    ("attention_tiles_singles", "attention_tiles_singles[attention]", "decode attention"),
    ("retention", "attention_tiles[attention] / attention_tiles_singles[attention]", "the other token mixer"),
    ("route_gated_act", "route_act", "routing + activation"),
    ("gated_act", None, "act(gate) * up of the dense feed-forward"),
)


def bimolix_config(size: str, layers: int):
    """Retention layers with a dense feed-forward and chunked attention layers with experts in turn: the
    experts as many and as wide as Kelasun's at this size."""
    from tinyvllm_b200.models import BimolixConfig
    from tinyvllm_b200.models.bimolix import BimolixFeedForward, BimolixLayer

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    unit = kelasun_expert_width(ff)
    experts = BimolixFeedForward(kind="moe", ff=unit, limit=7.0, experts=KELASUN_EXPERTS, top=KELASUN_TOP,
                                 route_scale=2.5, groups=4, keep=2, shared_ff=ff - KELASUN_TOP * unit, shared_limit=7.0)
    decay = tuple(1.0 - 2.0 ** -(5 + 4 * h / heads) for h in range(heads))
    made = []
    for index in range(layers):
        if index % 2 == 0:
            made.append(BimolixLayer(type="retention", heads=heads, dim=dim, vdim=dim, decay=decay, rot_dims=dim,
                                     rot_base=1000000.0, mlp=BimolixFeedForward(kind="dense", ff=ff)))
        else:
            made.append(BimolixLayer(type="attention", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                                     bias_max=float(BIMOLIX_CHUNK), chunk=BIMOLIX_CHUNK, mlp=experts,
                                     rel_rows=BIMOLIX_TABLE_ROWS))
    return BimolixConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, layers=tuple(made))


def bimolix_roofline(name: str, size: str, tokens: int, context: int, peak: dict):
    """(microseconds at the peaks, what bounds it) of one call of kernel ``name`` in a Bimolix layer:
    ``tokens`` new tokens whose requests hold ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    unit = kelasun_expert_width(ff)
    columns = KELASUN_EXPERTS * unit + (ff - KELASUN_TOP * unit)
    prompt = context == tokens
    bytes_, flops, fp32 = 0.0, 0.0, 0.0
    if name == "stream_norm":
        bytes_ = tokens * width * (4 + 4 + 4 + 2)
    elif name == "qkv_prepare":
        bytes_ = tokens * dim * 2 * ((heads + kv) * 2 + kv)          # q and k in place, k and the value copy to pages
    elif name == "attention_tiles":
        pairs = sum(p % BIMOLIX_CHUNK + 1 for p in range(tokens))
        flops = 2.0 * heads * 2 * dim * pairs
    elif name == "attention_tiles_singles":
        bytes_ = tokens * kv * (context % BIMOLIX_CHUNK + 1) * 2 * dim * 2
    elif name == "retention":
        fp32 = 4.0 * tokens * heads * dim * dim                      # state update and read-out, a multiply-add each
        bytes_ = (0 if prompt else tokens) * heads * dim * dim * 4 * 2 + tokens * heads * dim * 2 * 5
    elif name == "route_gated_act":
        bytes_ = tokens * columns * 2 * 3
    elif name == "gated_act":
        bytes_ = tokens * ff * 2 * 3
    if flops:
        return flops / (peak["bf16_tflops"] * 1e12) * 1e6, "tensor"
    by_memory = bytes_ / (peak["hbm_gbs"] * 1e9) * 1e6
    by_fp32 = fp32 / (FP32_TFLOPS_NOMINAL * 1e12) * 1e6
    return (by_fp32, "fp32 (nominal)") if by_fp32 > by_memory else (by_memory, "memory")


def bimolix_workload(args) -> int:
    """Prefill and decode of Bimolix at the layer sizes of the 0.6B, 8B and 32B models (random weights,
    ``--layers`` layers, default 4: retention layers with a dense feed-forward and attention layers in
    chunks of 1,024 with 8 experts of which 2 are used plus a shared one, in turn) beside Kelasun of the
    same sizes: tokens/s through the engine, and every kernel of both designs with the fraction of its
    roofline.  One JSON line."""
    import torch

    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepEntry

    layers = args.layers if args.layers_given else 4
    batch, prompt, steps, warmup = args.batch, PROMPT_TOKENS, min(args.steps, 64), max(args.warmup, 3)
    peak, peak_source = peaks()
    names = sorted({"stream_norm", "qkv_prepare", "attention_tiles", "attention_tiles_singles", "retention",
                    "route_gated_act", "gated_act", "attention_rows"}
                   | {n for pair in KELASUN_LIKE for n in pair[:1]})
    both_kinds = ("attention_tiles", "attention_tiles_singles", "attention_rows")
    results = []
    sampler = ClockSampler()
    sampler.start()
    sizes = [size for size in KELASUN_SIZES if not args.sizes or size in args.sizes.split(",")]
    for size in sizes:
        row = {"size": size}
        for label, config in (("bimolix", bimolix_config(size, layers)), ("kelasun", kelasun_config(size, layers))):
            with tempfile.TemporaryDirectory() as folder:
                Path(folder, "config.json").write_text(json.dumps(config.to_json()))
                engine = Engine.from_config(EngineConfig(
                    model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=CONTEXT_LIMIT,
                    max_num_seqs=batch, max_num_batched_tokens=4096, prefill_chunk_size=2048,
                    prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
                    kv_cache_memory_bytes=2 * 1024**3, graph_batch_sizes=(batch,)))
                decode = run_decode(engine, batch, steps, warmup, sampler, prompt_tokens=prompt)
                prefill_ms = run_prefill(engine, repeats=5, tokens=prompt)
                runner = engine.runner
                rng = random.Random(5)
                with torch.inference_mode():
                    for r in range(batch):
                        runner.open(f"k{r}")
                    prompts = [StepEntry(f"k{r}", tuple(random_prompt(rng, prompt)), ()) for r in range(batch)]

                    def eager_step(entries):
                        plan = runner.plan(entries)
                        runner.execute(runner.build_context(entries, plan))
                        runner.manager.commit(plan)

                    # the GPU is kept busy (a spin kernel) while the host queues the step's launches behind it:
                    # the events then bracket device time, not the host's pace
                    for entry in prompts[1:]:
                        eager_step([entry])
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step([prompts[0]])
                    torch.cuda.synchronize()
                    by_prompt = list(clock.marks)
                    singles = [StepEntry(f"k{r}", (1,), (0,)) for r in range(batch)]
                    eager_step(singles)
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step(singles)
                    torch.cuda.synchronize()
                    by_decode = list(clock.marks)
                    for r in range(batch):
                        runner.close(f"k{r}")
                kernels_out = {}
                for phase, marks, tokens in (("prefill", by_prompt, prompt), ("decode", by_decode, batch)):
                    found, seen = {}, {}
                    for name, start, end in marks:
                        kind = "bimolix"
                        if label == "kelasun":
                            index = seen.get(name, 0)
                            seen[name] = index + 1
                            kind = ("attention", "latent")[index % 2] if name in both_kinds else \
                                "latent" if name in ("latent_prepare", "rotate_heads", "head_product") else "attention"
                        key = name if label == "bimolix" or name not in both_kinds else f"{name}[{kind}]"
                        calls, ms, _ = found.get(key, (0, 0.0, kind))
                        found[key] = (calls + 1, ms + start.elapsed_time(end), kind)
                    for key, (calls, ms, kind) in sorted(found.items()):
                        per_call = 1e3 * ms / max(1, calls)
                        if label == "bimolix":
                            ideal, bound = bimolix_roofline(key, size, tokens, prompt, peak)
                        else:
                            ideal, bound = kelasun_roofline(key.split("[")[0], kind, size, tokens, prompt, peak)
                        kernels_out[f"{phase}:{key}"] = {
                            "calls": calls, "us_per_call": round(per_call, 2), "roofline_us": round(ideal, 2),
                            "bound": bound, "frac": round(ideal / per_call, 3) if per_call > 0 else None}
                row[label] = {
                    "decode_tokens_per_s": round(decode["tokens_per_s"], 1), "decode_ms_per_step": round(decode["ms_per_step"], 4),
                    "prefill_tokens_per_s": round(prompt / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                    "weight_bytes": engine.runner.model.weight_bytes(), "kernels": kernels_out}
                engine.close()
                del engine
                torch.cuda.empty_cache()
        results.append(row)
    sampler.stop()
    print(json.dumps({
        "metric": "Bimolix beside Kelasun of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "batch": batch, "vocab": MODEL["vocab_size"],
                   "sizes": {k: list(v) for k, v in KELASUN_SIZES.items() if k in sizes},
                   "chunk": BIMOLIX_CHUNK, "table_rows": BIMOLIX_TABLE_ROWS, "experts": KELASUN_EXPERTS,
                   "top": KELASUN_TOP, "like_kernels": [list(pair) for pair in BIMOLIX_LIKE],
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"],
                  "fp32_tflops_nominal": round(FP32_TFLOPS_NOMINAL, 1), "source": peak_source},
        "clocks": sampler.summary(), "results": results}))
    return 0


# ------------------------------------------- Fezavik beside Bimolix at equal layer sizes
FEZAVIK_WINDOW, FEZAVIK_IDENTITY = 1024, 2
# (kernel of the new design, its counterpart in Bimolix) by what they do
FEZAVIK_LIKE = (
    ("sandwich_norm", "stream_norm", "norm(s) around the residual sum"),
    ("projection_norm", "qkv_prepare", "q/k norm, rotation, cache write"),
    ("attention_tiles[attention]", "attention_tiles", "prompt attention"),
    ("attention_tiles_singles[attention]", "attention_tiles_singles", "decode attention"),
    ("attention_tiles[latent] / attention_tiles_singles[latent]", "attention_tiles / attention_tiles_singles",
     "attention over latent rows"),
    ("gated_recurrence", "retention", "the recurrent mixer"),
    ("route_softmax_gated", "route_gated_act", "routing + activation"),
)


def fezavik_config(size: str, layers: int):
    """Attention, recurrent and latent layers in turn, all with experts as many and as wide as Bimolix's at
    this size plus pass-through slots; windows of 1,024 keys."""
    from tinyvllm_b200.models import FezavikConfig
    from tinyvllm_b200.models.fezavik import FezavikExperts, FezavikLayer, FezavikRotation

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    q_rank, kv_rank = KELASUN_LATENTS[size]
    experts = FezavikExperts(experts=KELASUN_EXPERTS, top=KELASUN_TOP, ff=kelasun_expert_width(ff),
                             identity=FEZAVIK_IDENTITY)
    made = []
    for index in range(layers):
        if index % 3 == 0:
            made.append(FezavikLayer(type="attention", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                                     window=FEZAVIK_WINDOW, mlp=experts,
                                     rot=FezavikRotation(dims=dim // 2, base=1000000.0, scaling=(8.0, 1.0, 4.0, 8192.0))))
        elif index % 3 == 1:
            made.append(FezavikLayer(type="hgrn2", heads=heads, dim=dim, vdim=dim, mlp=experts))
        else:
            made.append(FezavikLayer(type="latent_attention", heads=heads, dim=dim // 2, rot_dim=KELASUN_ROT, vdim=dim,
                                     scale=dim ** -0.5, q_rank=q_rank, kv_rank=kv_rank, window=FEZAVIK_WINDOW,
                                     rot=FezavikRotation(dims=KELASUN_ROT, base=1000000.0), mlp=experts))
    return FezavikConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, layers=tuple(made))


def fezavik_roofline(name: str, kind: str, size: str, tokens: int, context: int, peak: dict):
    """(microseconds at the peaks, what bounds it) of one call of kernel ``name`` in a Fezavik layer of ``kind``:
    ``tokens`` new tokens whose requests hold ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    q_rank, kv_rank = KELASUN_LATENTS[size]
    row = kv_rank + KELASUN_ROT
    columns = KELASUN_EXPERTS * kelasun_expert_width(ff)
    prompt = context == tokens
    seen = lambda p: min(p + 1, FEZAVIK_WINDOW)                       # keys the query at position p attends
    pairs = sum(seen(p) for p in range(tokens)) if prompt else tokens * seen(context)
    bytes_, flops, fp32 = 0.0, 0.0, 0.0
    if name in ("sandwich_norm", "stream_norm"):
        bytes_ = tokens * width * (4 + 4 + 4 + 2)
    elif name == "projection_norm":
        # q, k and v read; q and k written where they stand, k and v to their pages (norm, rotation and store: one launch)
        bytes_ = tokens * dim * 2 * ((heads + 2 * kv) + (heads + 3 * kv))
    elif name == "qkv_prepare":
        bytes_ = tokens * dim * 2 * ((heads + kv) * 2 + 2 * kv)
    elif name == "latent_prepare":
        bytes_ = tokens * (q_rank + row) * 2 * 2
    elif name == "rotate_heads":
        bytes_ = tokens * heads * KELASUN_ROT * 2 * 2
    elif name == "head_product":
        flops = 2.0 * tokens * heads * kv_rank * (dim // 2 + dim) / 2
    elif name == "attention_tiles":
        flops = 2.0 * heads * ((row + kv_rank) if kind == "latent" else 2 * dim) * pairs
    elif name == "attention_tiles_singles":
        bytes_ = pairs * 2 * (row if kind == "latent" else kv * 2 * dim)
    elif name == "gated_recurrence":
        fp32 = 4.0 * tokens * heads * dim * dim
        bytes_ = (0 if prompt else tokens) * heads * dim * dim * 4 * 2 + tokens * heads * dim * 2 * 4
    elif name == "route_softmax_gated":
        bytes_ = tokens * columns * 2 * 3
    if flops:
        return flops / (peak["bf16_tflops"] * 1e12) * 1e6, "tensor"
    by_memory = bytes_ / (peak["hbm_gbs"] * 1e9) * 1e6
    by_fp32 = fp32 / (FP32_TFLOPS_NOMINAL * 1e12) * 1e6
    return (by_fp32, "fp32 (nominal)") if by_fp32 > by_memory else (by_memory, "memory")


def fezavik_workload(args) -> int:
    """Prefill and decode of Fezavik at the layer sizes of the 0.6B, 8B and 32B models (random weights,
    ``--layers`` layers, default 6: attention, recurrent and latent layers in turn, windows of 1,024 keys, 8
    experts of which 2 slots are used, 2 pass-through slots) beside Bimolix of the same sizes and depth: tokens/s
    through the engine, and every kernel of both designs with the fraction of its roofline.  One JSON line."""
    import torch

    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepEntry

    layers = args.layers if args.layers_given else 6
    batch, prompt, steps, warmup = args.batch, PROMPT_TOKENS, min(args.steps, 64), max(args.warmup, 3)
    peak, peak_source = peaks()
    names = sorted({"stream_norm", "sandwich_norm", "projection_norm", "qkv_prepare", "latent_prepare", "rotate_heads",
                    "head_product", "attention_tiles", "attention_tiles_singles", "attention_rows", "gated_recurrence",
                    "route_softmax_gated", "retention", "route_gated_act", "gated_act"})
    attending = ("attention_tiles", "attention_tiles_singles", "attention_rows")
    results = []
    sampler = ClockSampler()
    sampler.start()
    sizes = [size for size in KELASUN_SIZES if not args.sizes or size in args.sizes.split(",")]
    for size in sizes:
        row = {"size": size}
        for label, config in (("fezavik", fezavik_config(size, layers)), ("bimolix", bimolix_config(size, layers))):
            with tempfile.TemporaryDirectory() as folder:
                Path(folder, "config.json").write_text(json.dumps(config.to_json()))
                engine = Engine.from_config(EngineConfig(
                    model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=CONTEXT_LIMIT,
                    max_num_seqs=batch, max_num_batched_tokens=4096, prefill_chunk_size=2048,
                    prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
                    kv_cache_memory_bytes=2 * 1024**3, graph_batch_sizes=(batch,)))
                decode = run_decode(engine, batch, steps, warmup, sampler, prompt_tokens=prompt)
                prefill_ms = run_prefill(engine, repeats=5, tokens=prompt)
                runner = engine.runner
                rng = random.Random(5)
                with torch.inference_mode():
                    for r in range(batch):
                        runner.open(f"k{r}")
                    prompts = [StepEntry(f"k{r}", tuple(random_prompt(rng, prompt)), ()) for r in range(batch)]

                    def eager_step(entries):
                        plan = runner.plan(entries)
                        runner.execute(runner.build_context(entries, plan))
                        runner.manager.commit(plan)

                    for entry in prompts[1:]:
                        eager_step([entry])
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step([prompts[0]])
                    torch.cuda.synchronize()
                    by_prompt = list(clock.marks)
                    singles = [StepEntry(f"k{r}", (1,), (0,)) for r in range(batch)]
                    eager_step(singles)
                    torch.cuda.synchronize()
                    with KernelClock(names) as clock:
                        torch.cuda._sleep(40_000_000)
                        eager_step(singles)
                    torch.cuda.synchronize()
                    by_decode = list(clock.marks)
                    for r in range(batch):
                        runner.close(f"k{r}")
                kernels_out = {}
                for phase, marks, tokens in (("prefill", by_prompt, prompt), ("decode", by_decode, batch)):
                    found, kind = {}, "attention"
                    for name, start, end in marks:
                        if label == "fezavik":
                            # the layer a call belongs to: the latent layers prepare their rows first
                            if name in ("projection_norm", "qkv_prepare"):
                                kind = "attention"
                            elif name == "latent_prepare":
                                kind = "latent"
                        key = f"{name}[{kind}]" if label == "fezavik" and name in attending else name
                        calls, ms, _ = found.get(key, (0, 0.0, kind))
                        found[key] = (calls + 1, ms + start.elapsed_time(end), kind)
                    for key, (calls, ms, kind) in sorted(found.items()):
                        per_call = 1e3 * ms / max(1, calls)
                        if label == "fezavik":
                            ideal, bound = fezavik_roofline(key.split("[")[0], kind, size, tokens, prompt, peak)
                        else:
                            ideal, bound = bimolix_roofline(key, size, tokens, prompt, peak)
                        kernels_out[f"{phase}:{key}"] = {
                            "calls": calls, "us_per_call": round(per_call, 2), "roofline_us": round(ideal, 2),
                            "bound": bound, "frac": round(ideal / per_call, 3) if per_call > 0 else None}
                row[label] = {
                    "decode_tokens_per_s": round(decode["tokens_per_s"], 1), "decode_ms_per_step": round(decode["ms_per_step"], 4),
                    "prefill_tokens_per_s": round(prompt / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                    "weight_bytes": engine.runner.model.weight_bytes(), "kernels": kernels_out}
                engine.close()
                del engine
                torch.cuda.empty_cache()
        results.append(row)
    sampler.stop()
    print(json.dumps({
        "metric": "Fezavik beside Bimolix of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "batch": batch, "vocab": MODEL["vocab_size"],
                   "sizes": {k: list(v) for k, v in KELASUN_SIZES.items() if k in sizes},
                   "latents": {k: list(v) for k, v in KELASUN_LATENTS.items() if k in sizes},
                   "window": FEZAVIK_WINDOW, "experts": KELASUN_EXPERTS, "identity": FEZAVIK_IDENTITY,
                   "top": KELASUN_TOP, "like_kernels": [list(pair) for pair in FEZAVIK_LIKE],
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"],
                  "fp32_tflops_nominal": round(FP32_TFLOPS_NOMINAL, 1), "source": peak_source},
        "clocks": sampler.summary(), "results": results}))
    return 0


# ------------------------------------------- Zifunex beside Bimolix at equal layer sizes
ZIFUNEX_STREAMS, ZIFUNEX_STATE, ZIFUNEX_TAPS = 4, 16, 4
EXP_RATE_NOMINAL = 148 * 16 * 1.965e9                 # 2^x a second of the SMs' special-function units
# (kernel of the new design, its counterpart in Bimolix) by what they do
ZIFUNEX_LIKE = (
    ("hyper_norm", "stream_norm", "norm + residual write"),
    ("qkv_prepare", "qkv_prepare", "q/k/v bias, rotation or norm, cache write"),
    ("attention_tiles", "attention_tiles", "prompt attention"),
    ("attention_tiles_singles", "attention_tiles_singles", "decode attention"),
    ("gated_recurrence", "retention", "linear attention"),
    ("selective_scan", "retention", "the other recurrence"),
    ("short_convolution", "gated_act", "a pass over the activations"),
    ("gated_act", "gated_act", "act(gate) * up"),
)


def zifunex_config(size: str, layers: int):
    """Two layers with attention and a selective scan side by side (the scan twice the width, 16 numbers a
    channel), then one of gated linear attention, in turn; a dense feed-forward in every layer, four streams."""
    from tinyvllm_b200.models import ZifunexConfig
    from tinyvllm_b200.models.zifunex import (ZifunexAttention, ZifunexBigram, ZifunexLayer, ZifunexLinearAttention,
                                              ZifunexScan)

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    left = ZifunexAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, softcap=30.0,
                            rot_dims=dim, rot_base=1000000.0)
    right = ZifunexScan(inner=2 * width, state=ZIFUNEX_STATE, dt_rank=width // 16, conv=ZIFUNEX_TAPS)
    made = []
    for index in range(layers):
        if index % 3 == 2:
            made.append(ZifunexLayer(linear=ZifunexLinearAttention(heads=heads, dim=dim, vdim=dim, tau=12.0), ff=ff))
        else:
            made.append(ZifunexLayer(left=left, right=right, ff=ff))
    return ZifunexConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, streams=ZIFUNEX_STREAMS,
                         bigram=ZifunexBigram(buckets=65521, mul_prev=31, mul_cur=11), layers=tuple(made))


def dense_bimolix_config(size: str, layers: int):
    """Bimolix with its attention and retention layers in Zifunex's proportion and a dense feed-forward everywhere."""
    from tinyvllm_b200.models import BimolixConfig
    from tinyvllm_b200.models.bimolix import BimolixFeedForward

    retention, attention = bimolix_config(size, 2).layers
    dense = BimolixFeedForward(kind="dense", ff=KELASUN_SIZES[size][4])
    made = tuple(dataclasses.replace(retention if index % 3 == 2 else attention, mlp=dense) for index in range(layers))
    return BimolixConfig(vocab=MODEL["vocab_size"], width=KELASUN_SIZES[size][0], norm_eps=1e-6, layers=made)


def zifunex_roofline(name: str, size: str, tokens: int, context: int, peak: dict):
    """(microseconds at the peaks, what bounds it) of one call of kernel ``name`` in a Zifunex layer: ``tokens``
    new tokens whose requests hold ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    inner, state, prompt = 2 * width, ZIFUNEX_STATE, context == tokens
    bytes_, limits = 0.0, []
    if name == "hyper_norm":
        # streams read and written, the sublayer's float32 output (two of them behind the mixers side by side: two
        # of six writes in three layers), the normed row
        bytes_ = tokens * width * (ZIFUNEX_STREAMS * 4 * 2 + 4 * 8 / 6 + 2)
    elif name == "qkv_prepare":
        bytes_ = tokens * dim * 2 * ((heads + 2 * kv) + (heads + 2 * kv))
    elif name == "attention_tiles":
        limits.append((2.0 * heads * 2 * dim * tokens * (tokens + 1) / 2 / (peak["bf16_tflops"] * 1e12), "tensor"))
    elif name == "attention_tiles_singles":
        bytes_ = tokens * kv * (context + 1) * 2 * dim * 2
    elif name == "short_convolution":
        bytes_ = tokens * inner * 2 * 2 + (0 if prompt else tokens * inner * (ZIFUNEX_TAPS - 1) * 4 * 2)
    elif name == "selective_scan":
        bytes_ = tokens * (inner * (2 + 4 + 2 + 2) + 4 * state) + (0 if prompt else tokens) * inner * state * 4 * 2
        limits.append((tokens * inner * state / EXP_RATE_NOMINAL, "2^x (nominal)"))
    elif name == "gated_recurrence":
        bytes_ = (0 if prompt else tokens) * heads * dim * dim * 4 * 2 + tokens * heads * dim * 2 * 5
        limits.append((4.0 * tokens * heads * dim * dim / (FP32_TFLOPS_NOMINAL * 1e12), "fp32 (nominal)"))
    elif name == "gated_act":
        bytes_ = tokens * ff * 2 * 3
    elif name == "embed_pairs":
        bytes_ = tokens * width * (2 + 2 + 4)
    limits.append((bytes_ / (peak["hbm_gbs"] * 1e9), "memory"))
    seconds, bound = max(limits)
    return seconds * 1e6, bound


def measure_design(config, names, batch: int, prompt: int, steps: int, warmup: int, sampler):
    """A model of ``config`` with random weights through the engine: decode and prefill figures, and the CUDA-event
    marks of every call of the kernels ``names`` in one prompt step and one decode step."""
    import torch

    from tinyvllm_b200 import EngineConfig
    from tinyvllm_b200.engine.engine import Engine
    from tinyvllm_b200.engine.step import StepEntry

    with tempfile.TemporaryDirectory() as folder:
        Path(folder, "config.json").write_text(json.dumps(config.to_json()))
        engine = Engine.from_config(EngineConfig(
            model=folder, dtype="bfloat16", weights="random", seed=0, max_model_len=CONTEXT_LIMIT,
            max_num_seqs=batch, max_num_batched_tokens=4096, prefill_chunk_size=2048,
            prefill_reserve_tokens=0, prefill_reserve_requests=0, kv_block_size=16,
            kv_cache_memory_bytes=2 * 1024**3, graph_batch_sizes=(batch,)))
    decode = run_decode(engine, batch, steps, warmup, sampler, prompt_tokens=prompt)
    prefill_ms = run_prefill(engine, repeats=5, tokens=prompt)
    runner = engine.runner
    rng = random.Random(5)
    with torch.inference_mode():
        for r in range(batch):
            runner.open(f"k{r}")
        prompts = [StepEntry(f"k{r}", tuple(random_prompt(rng, prompt)), ()) for r in range(batch)]

        def eager_step(entries, timed: bool):
            plan = runner.plan(entries)
            ctx = runner.build_context(entries, plan)
            torch.cuda.synchronize()
            marks = []
            if timed:
                # the GPU is kept busy (a spin kernel) while the host queues the step's launches behind it:
                # the events then bracket device time, not the host's pace
                with KernelClock(names) as clock:
                    torch.cuda._sleep(40_000_000)
                    runner.execute(ctx)
                marks = list(clock.marks)
            else:
                runner.execute(ctx)
            torch.cuda.synchronize()
            runner.manager.commit(plan)
            return marks

        for entry in prompts[1:]:
            eager_step([entry], False)
        by_prompt = eager_step([prompts[0]], True)
        singles = [StepEntry(f"k{r}", (1,), (0,)) for r in range(batch)]
        eager_step(singles, False)
        by_decode = eager_step(singles, True)
        for r in range(batch):
            runner.close(f"k{r}")
    weight_bytes = runner.model.weight_bytes()
    engine.close()
    del engine, runner
    torch.cuda.empty_cache()
    return decode, prefill_ms, by_prompt, by_decode, weight_bytes


def zifunex_workload(args) -> int:
    """Prefill and decode of Zifunex at the layer sizes of the 0.6B, 8B and 32B models (random weights,
    ``--layers`` layers, default 6) beside Bimolix of the same sizes and depth, both with a dense feed-forward in
    every layer: tokens/s through the engine, and every kernel of both designs with the fraction of its roofline.
    One JSON line."""
    layers = args.layers if args.layers_given else 6
    batch, prompt = args.batch, PROMPT_TOKENS
    peak, peak_source = peaks()
    names = ("hyper_norm", "stream_norm", "qkv_prepare", "attention_tiles", "attention_tiles_singles", "attention_rows",
             "gated_recurrence", "retention", "selective_scan", "short_convolution", "gated_act", "embed_pairs")
    sizes, results, clocks = designs_side_by_side(args, names, peak, {
        "zifunex": (lambda size: zifunex_config(size, layers), zifunex_roofline),
        "bimolix": (lambda size: dense_bimolix_config(size, layers), bimolix_roofline)})
    print(json.dumps({
        "metric": "Zifunex beside Bimolix of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "batch": batch, "vocab": MODEL["vocab_size"],
                   "sizes": {k: list(v) for k, v in KELASUN_SIZES.items() if k in sizes},
                   "streams": ZIFUNEX_STREAMS, "scan_state": ZIFUNEX_STATE, "taps": ZIFUNEX_TAPS,
                   "like_kernels": [list(pair) for pair in ZIFUNEX_LIKE],
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"],
                  "fp32_tflops_nominal": round(FP32_TFLOPS_NOMINAL, 1), "exp_per_s_nominal": EXP_RATE_NOMINAL,
                  "source": peak_source},
        "clocks": clocks, "results": results}))
    return 0


def designs_side_by_side(args, names, peak: dict, designs: dict):
    """Every size's designs (label -> (size -> configuration, roofline)) measured one after the other with
    :func:`measure_design`: (sizes, a row a size, clocks seen)."""
    batch, prompt, steps, warmup = args.batch, PROMPT_TOKENS, min(args.steps, 64), max(args.warmup, 3)
    results = []
    sampler = ClockSampler()
    sampler.start()
    sizes = [size for size in KELASUN_SIZES if not args.sizes or size in args.sizes.split(",")]
    for size in sizes:
        row = {"size": size}
        for label, (config_of, roofline) in designs.items():
            config = config_of(size)
            decode, prefill_ms, by_prompt, by_decode, weight_bytes = measure_design(
                config, names, batch, prompt, steps, warmup, sampler)
            kernels_out = {}
            for phase, marks, tokens in (("prefill", by_prompt, prompt), ("decode", by_decode, batch)):
                found = {}
                for name, start, end in marks:
                    calls, ms = found.get(name, (0, 0.0))
                    found[name] = (calls + 1, ms + start.elapsed_time(end))
                for name, (calls, ms) in sorted(found.items()):
                    per_call = 1e3 * ms / calls
                    ideal, bound = roofline(name, size, tokens, prompt, peak)
                    kernels_out[f"{phase}:{name}"] = {
                        "calls": calls, "us_per_call": round(per_call, 2), "roofline_us": round(ideal, 2),
                        "bound": bound, "frac": round(ideal / per_call, 3) if per_call > 0 else None}
            row[label] = {
                "decode_tokens_per_s": round(decode["tokens_per_s"], 1), "decode_ms_per_step": round(decode["ms_per_step"], 4),
                "prefill_tokens_per_s": round(prompt / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
                "weight_bytes": weight_bytes, "kernels": kernels_out}
        results.append(row)
    sampler.stop()
    return sizes, results, sampler.summary()


# ------------------------------------------- Lasupel beside Bimolix at equal layer sizes
LASUPEL_WINDOW, LASUPEL_TAPS = 1024, 4
# (kernel of the new design, its counterpart in Bimolix) by what they do
LASUPEL_LIKE = (
    ("sandwich_norm", "stream_norm", "norm + residual sum"),
    ("qkv_prepare", "qkv_prepare", "q/k norm, rotation or bias, cache write"),
    ("attention_tiles", "attention_tiles", "prompt attention"),
    ("attention_tiles_singles", "attention_tiles_singles", "decode attention"),
    ("delta_rule", "retention", "linear attention"),
    ("recurrent_unit", "retention", "the other recurrence"),
    ("block_products", None, "the recurrent unit's gates (a library product)"),
    ("short_convolution", "gated_act", "a pass over the activations"),
    ("route_softmax_gated", "route_gated_act", "routing + activation"),
    ("gated_act", "gated_act", "act(gate) * up"),
)


def lasupel_config(size: str, layers: int):
    """A recurrent unit as wide as the model, attention over a window of 1,024 keys, a delta rule with two value heads a
    key head, and attention that reads the keys of the layer two before, in turn; recurrent layers with a dense
    feed-forward, attention layers with experts as many and as wide as Bimolix's at this size."""
    from tinyvllm_b200.models import LasupelConfig
    from tinyvllm_b200.models.lasupel import (LasupelAttention, LasupelDelta, LasupelFeedForward, LasupelLayer,
                                              LasupelRecurrentUnit)

    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    dense = LasupelFeedForward(kind="dense", ff=ff)
    experts = LasupelFeedForward(kind="moe", ff=kelasun_expert_width(ff), limit=7.0, experts=KELASUN_EXPERTS, top=KELASUN_TOP,
                                 groups=4, keep=2)
    made = []
    for index in range(layers):
        attention = LasupelAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, window=LASUPEL_WINDOW,
                                     rot_dims=dim // 2, rot_base=1000000.0, kv_from=index - 2 if index % 4 == 3 else None)
        if index % 2 == 1:
            made.append(LasupelLayer(attention, experts))
        elif index % 4 == 0:
            made.append(LasupelLayer(LasupelRecurrentUnit(width=width, blocks=heads, conv=LASUPEL_TAPS), dense))
        else:
            made.append(LasupelLayer(LasupelDelta(heads=heads, kv_heads=heads // 2, dim=dim, vdim=dim, conv=LASUPEL_TAPS), dense))
    return LasupelConfig(vocab=MODEL["vocab_size"], width=width, norm_eps=1e-6, embedding_scale=width ** 0.5, layers=tuple(made))


def lasupel_roofline(name: str, size: str, tokens: int, context: int, peak: dict):
    """(microseconds at the peaks, what bounds it) of one call of kernel ``name`` in a Lasupel layer: ``tokens``
    new tokens whose requests hold ``context`` tokens each (a prompt: context == tokens)."""
    width, heads, kv, dim, ff = KELASUN_SIZES[size]
    prompt, part = context == tokens, width // heads
    seen = lambda p: min(p + 1, LASUPEL_WINDOW)                       # keys the query at position p attends
    bytes_, limits = 0.0, []
    if name == "sandwich_norm":
        bytes_ = tokens * width * (4 + 4 + 4 + 2)
    elif name == "qkv_prepare":
        # q in place in every attention layer; k and v to their pages in every other one
        bytes_ = tokens * dim * 2 * (2 * heads + 4 * kv / 2)
    elif name == "attention_tiles":
        limits.append((2.0 * heads * 2 * dim * sum(seen(p) for p in range(tokens)) / (peak["bf16_tflops"] * 1e12), "tensor"))
    elif name == "attention_tiles_singles":
        bytes_ = tokens * kv * seen(context) * 2 * dim * 2
    elif name == "short_convolution":                                 # of the unit and of the delta rule in turn
        bytes_ = tokens * (width + 2 * heads * dim) / 2 * (2 * 2 + (0 if prompt else (LASUPEL_TAPS - 1) * 4 * 2))
    elif name == "recurrent_unit":
        # u, y, the result and the gates' pre-activations (few requests: the gates' weights instead), the state twice
        from tinyvllm_b200.ops import kernels
        inside = not prompt and kernels.recurrent_unit_step_takes(tokens, part)
        bytes_ = tokens * width * (2 + 2 + 2 + (0 if inside else 8) + (0 if prompt else 8)) + (2 * width * part * 2 if inside else 0)
    elif name == "block_products":
        bytes_ = tokens * width * (2 + 8) + 2 * width * part * 2
        limits.append((2.0 * tokens * width * 2 * part / (peak["bf16_tflops"] * 1e12), "tensor"))
    elif name == "delta_rule":
        # read under the key, write, read-out: a multiply-add each
        limits.append((6.0 * tokens * heads * dim * dim / (FP32_TFLOPS_NOMINAL * 1e12), "fp32 (nominal)"))
        bytes_ = (0 if prompt else tokens) * heads * dim * dim * 4 * 2 + tokens * heads * dim * 2 * 4
    elif name == "route_softmax_gated":
        bytes_ = tokens * KELASUN_EXPERTS * kelasun_expert_width(ff) * 2 * 3
    elif name == "gated_act":
        bytes_ = tokens * ff * 2 * 3
    elif name == "embed_scaled":
        bytes_ = tokens * width * (2 + 4 + 2)
    limits.append((bytes_ / (peak["hbm_gbs"] * 1e9), "memory"))
    seconds, bound = max(limits)
    return seconds * 1e6, bound


def lasupel_workload(args) -> int:
    """Prefill and decode of Lasupel at the layer sizes of the 0.6B, 8B and 32B models (random weights,
    ``--layers`` layers, default 4) beside Bimolix of the same sizes, depth and feed-forwards: tokens/s through the
    engine, and every kernel of both designs with the fraction of its roofline.  One JSON line."""
    layers = args.layers if args.layers_given else 4
    batch, prompt = args.batch, PROMPT_TOKENS
    peak, peak_source = peaks()
    names = ("sandwich_norm", "stream_norm", "qkv_prepare", "attention_tiles", "attention_tiles_singles", "attention_rows",
             "delta_rule", "retention", "recurrent_unit", "block_products", "short_convolution", "route_softmax_gated",
             "route_gated_act", "gated_act", "embed_scaled")
    sizes, results, clocks = designs_side_by_side(args, names, peak, {
        "lasupel": (lambda size: lasupel_config(size, layers), lasupel_roofline),
        "bimolix": (lambda size: bimolix_config(size, layers), bimolix_roofline)})
    print(json.dumps({
        "metric": "Lasupel beside Bimolix of equal layer sizes: decode tok/s at batch "
                  f"{batch} from context {prompt:,}, prefill tok/s of {prompt:,} tokens, bf16",
        "unit": "tokens/s", "n_gpus": 1, "dtype": "bf16", "data": "synthetic (random weights and tokens)",
        "config": {"layers": layers, "batch": batch, "vocab": MODEL["vocab_size"],
                   "sizes": {k: list(v) for k, v in KELASUN_SIZES.items() if k in sizes},
                   "window": LASUPEL_WINDOW, "taps": LASUPEL_TAPS, "experts": KELASUN_EXPERTS, "top": KELASUN_TOP,
                   "like_kernels": [list(pair) for pair in LASUPEL_LIKE],
                   "timing": "CUDA events; decode replays graphs with inputs uploaded every step, for "
                             f"{batch} requests; kernel figures: the calls of one eager step queued behind a spin kernel, "
                             "so that each pair of events brackets device time (warm caches)"},
        "peaks": {"hbm_gbs": peak["hbm_gbs"], "bf16_tflops": peak["bf16_tflops"],
                  "fp32_tflops_nominal": round(FP32_TFLOPS_NOMINAL, 1), "source": peak_source},
        "clocks": clocks, "results": results}))
    return 0


def arrivals_workload(args) -> int:
    """16 requests with prompts of 64 or 512 tokens and 64 new tokens that arrive 20 ms apart, at the
    0.6B sizes, through ``Engine.submit(arrival_ns=)`` and ``Engine.step``: time to first token, time
    per output token and output tokens per second."""
    import torch

    from tinyvllm_b200 import SamplingParams

    requests, new, gap_ns = 16, 64, 20_000_000
    rng = random.Random(16)
    with tempfile.TemporaryDirectory() as folder:
        engine = make_engine(folder, args.layers, requests, new_tokens=new)
        prompts = [random_prompt(rng, 64 if index % 2 == 0 else 512) for index in range(requests)]
        sampling = SamplingParams(max_new_tokens=new, ignore_eos=True)
        results = []
        for _ in range(3):                             # the first pass settles graphs and allocations
            torch.cuda.synchronize()
            origin = time.monotonic_ns()
            ids = [engine.submit(prompt, sampling, arrival_ns=origin + index * gap_ns)
                   for index, prompt in enumerate(prompts)]
            done = {}
            while engine.has_unfinished():
                events = engine.step()
                for output in events.finished:
                    done[output.request_id] = output
                if not events.tokens and not events.finished:
                    ahead = engine.scheduler.next_arrival_ns
                    if ahead is not None:
                        time.sleep(max(0.0, (ahead - time.monotonic_ns()) / 1e9))
            torch.cuda.synchronize()
            finish = max(done[i].finished_ns for i in ids)
            ttft = [(done[i].first_token_ns - done[i].arrival_ns) / 1e6 for i in ids]
            tpot = [(done[i].finished_ns - done[i].first_token_ns) / 1e6 / (new - 1) for i in ids]
            results.append({"ttft_ms": statistics.mean(ttft), "tpot_ms": statistics.mean(tpot),
                            "tokens_per_s": requests * new / ((finish - origin) / 1e9)})
        engine.close()
    best = results[-1]
    print(json.dumps({
        "metric": "arrivals: 16 requests, 64/512 -> 64 tokens, 20 ms apart (Qwen3-0.6B dims, bf16)",
        "value": round(best["tokens_per_s"], 1), "unit": "tokens/s", "n_gpus": 1, "higher_is_better": True,
        "dtype": "bf16", "impl": "ours", "ttft_ms": round(best["ttft_ms"], 3), "tpot_ms": round(best["tpot_ms"], 3),
        "passes": [{k: round(v, 3) for k, v in r.items()} for r in results],
        "data": "synthetic: uniform random token ids, random weights N(0, 0.02)",
        "config": {"model": "Qwen3-0.6B dims", "layers": args.layers, "requests": requests, "new_tokens": new,
                   "arrival_gap_ms": 20, "note": "the arrival schedule bounds tokens/s from above"}}))
    return 0


def main() -> int:
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=256)
    parser.add_argument("--warmup", type=int, default=8)
    parser.add_argument("--impl", choices=("ours", "reference"), default="ours")
    parser.add_argument("--workload", choices=("0.6b", "8b", "32b", "arrivals", "gumapel", "kelasun", "bimolix", "fezavik",
                                               "zifunex", "lasupel"),
                        default="0.6b",
                        help="0.6b: the decode and prefill measurement (default); 8b, 32b: the serving "
                             "workloads of those sizes at full depth; arrivals: 16 requests 20 ms apart; "
                             "gumapel: the Gumapel design beside a windowed Qwen3 at equal layer sizes; "
                             "kelasun: the Kelasun design beside a dense Qwen3 at equal layer sizes; "
                             "bimolix: the Bimolix design beside Kelasun at equal layer sizes; "
                             "fezavik, zifunex, lasupel: those designs beside Bimolix at equal layer sizes")
    parser.add_argument("--sizes", default="", help="kelasun, bimolix, fezavik, zifunex, lasupel: which of 0.6b,8b,32b (default: all)")
    parser.add_argument("--layers", type=int, default=None,
                        help="fewer layers than the configuration has (both numbers are in the line)")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--no-points", action="store_true", help="skip batch 1 and 64")
    parser.add_argument("--eager-profile", action="store_true",
                        help="no graphs: run warm-up + steps decode steps and one prefill kernel by "
                             "kernel, for a profiler; prints no bench line")
    args = parser.parse_args()
    args.layers_given = args.layers is not None
    if args.layers is None:
        args.layers = MODEL["num_hidden_layers"]
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not built (this engine is single-GPU)")
        return 2
    if args.impl == "reference":
        return reference_arm(args)
    sys.path.insert(0, str(ROOT))
    warmup = max(args.warmup, 3)
    if args.workload in SERVING:
        return serving_workload(args)
    if args.workload == "arrivals":
        return arrivals_workload(args)
    if args.workload == "gumapel":
        return gumapel_workload(args)
    if args.workload == "kelasun":
        return kelasun_workload(args)
    if args.workload == "bimolix":
        return bimolix_workload(args)
    if args.workload == "fezavik":
        return fezavik_workload(args)
    if args.workload == "zifunex":
        return zifunex_workload(args)
    if args.workload == "lasupel":
        return lasupel_workload(args)
    if args.eager_profile:
        return eager_profile(args, warmup)
    return headline(args, warmup)


if __name__ == "__main__":
    sys.exit(main())
