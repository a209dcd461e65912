"""Decode and prefill throughput of Qwen3 shapes with random weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--shape 4b|8b|0.6b] [--impl ours|reference]
                    [--batch B] [--layers L] [--skip-points] [--skip-kernels]
    python bench.py --design lopazen [--sizes 0.6b,4b,1b-h64] [--layers L] [--batch B] [--skip-kernels]
    python bench.py --design susalorn [--sizes 1b,2b-dense] [--layers L] [--batch B] [--skip-kernels]
    python bench.py --design bolelix [--sizes 1b,2b] [--layers L] [--batch B] [--skip-kernels]
    python bench.py --design musavik [--sizes 1b,2b] [--layers L] [--batch B] [--skip-kernels]
    python bench.py --design kamosun [--sizes 1b,2b] [--layers L] [--batch B] [--skip-kernels]
    python bench.py --design gesuvik [--sizes 1b,2b] [--layers L] [--batch B] [--skip-kernels]

The shapes and workloads are the ones BASELINE.json names (its configs[2], [3], [4]):

4b    (default) batch 8, 2,048-token prompts, context limit 4,096; decode at batch 1 and 64 and a
      prefill of 2,048 tokens beside it
8b    a ragged batch of 16 prompts with seeded lengths U[64, 2048], then 256 decode steps, untied head
0.6b  batch 64 with caches of 8,192 tokens

A step is one decode step of the batch.  ``value`` is decoded tokens per second over K replays of
the captured step timed with CUDA events, repeated until at least a second of device time has
been timed (``repeats``).  ``e2e`` times whole ``Engine.generate`` calls the way the reference's
own harness does (bench/bench.py:30-38, 61-75): host token lists in, the prompt step and every
decode step inside the clock, every step's tokens read back on the host; it gives tokens per
second of the whole call, the time to the first token, and the rate after the first token.
``prefill`` is one 2,048-token prompt; ``roofline`` divides the bytes a decode step has to read
(each weight once plus the live cache) by its time; ``kernels`` times each kernel of the decode
step and of the prompt step on its own (:mod:`enginekernel_b200.measure`) against the measured
peaks.  ``--design lopazen`` leaves that workload alone and instead measures the Lopazen decoder
beside the Qwen3 decoder at equal layer sizes (12 layers unless ``--layers`` says otherwise): a
2,048-token prompt step, decode steps of a batch of 8, and both per-kernel tables for each.
``--design susalorn`` does the same for the Susalorn decoder (alternating latent-attention and
delta-rule layers over four residual streams, routed or dense feed-forwards) beside a Qwen3 decoder
of the same width, layer count and feed-forward work per token.
``--design bolelix`` measures the Bolelix decoder (state-space, windowed-attention and matrix-memory layers in
turn, every one with gated routed experts beside the mixer) next to the Susalorn decoder of the same width, layer
count and experts.
``--design musavik`` measures the Musavik decoder (two gated linear recurrences, then attention with mixed heads
beside a delta rule, every layer with norms on both sides of its sublayers and a dense feed-forward) next to the
Bolelix decoder of the same width and layer count.
``--design kamosun`` measures the Kamosun decoder (a pair of full attention and fixed-decay memory, then three layers of
chunked attention, one of which reads another's keys, all with gated results, averages over the depth and routed
experts beside a shared one) next to the Bolelix decoder of the same width, layer count and experts.
``--design gesuvik`` measures the Gesuvik decoder (retention, windowed latent attention, retention and windowed
attention in turn, every one with routed experts, some of them the identity, beside a shared one) next to the Kamosun
decoder of the same width, layer count, heads and experts.
One line of JSON is printed.  The inputs of a step (gigabytes of weights) are larger than
the L2.

``--impl reference`` runs the unmodified reference from ``baseline/_ref`` (a plain copy of its
tree) on the same workload: its stock ``Engine(model_path).generate(input_ids, max_new_tokens)``
(engine/engine.py:770-830) on a folder of random weights of the same shape, with none of this
repository's kernels, models or engine on that path.
"""

from __future__ import annotations

import argparse
import json
import math
import os
import re
import shutil
import statistics
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

# What BASELINE.json's configs say, kept here for runs without that file; re-read from it when it
# is there.  (index in "configs", sizes, workload)
SHAPES = {
    "4b": (2, {"num_hidden_layers": 36, "hidden_size": 2560, "num_attention_heads": 32,
               "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 9728,
               "vocab_size": 151936, "rope_theta": 5000000.0, "rms_norm_eps": 1e-6,
               "tie_word_embeddings": True, "max_position_embeddings": 4096},
           {"batch": 8, "prompt": 2048, "context": 4096, "steps": 128, "name": "Qwen3-4B"}),
    "8b": (3, {"num_hidden_layers": 36, "hidden_size": 4096, "num_attention_heads": 32,
               "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 12288,
               "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6,
               "tie_word_embeddings": False, "max_position_embeddings": 4096},
           {"batch": 16, "prompt": (64, 2048), "context": 4096, "steps": 256, "name": "Qwen3-8B"}),
    "0.6b": (4, {"num_hidden_layers": 28, "hidden_size": 1024, "num_attention_heads": 16,
                 "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 3072,
                 "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6,
                 "tie_word_embeddings": True, "max_position_embeddings": 8192},
             {"batch": 64, "prompt": 7936, "context": 8192, "steps": 64, "name": "Qwen3-0.6B"}),
}
PREFILL_TOKENS = 2048
MIN_TIMED_SECONDS = 1.0
STEP_BUDGET = 900                  # decode steps a timed batch may take in all (keeps its context bucket)
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def shape_config(shape: str = "4b"):
    index, preset, _ = SHAPES[shape]
    cfg = dict(preset)
    try:
        with open(os.path.join(ROOT, "BASELINE.json")) as f:
            text = json.load(f)["configs"][index]
        for key, cast in (("num_hidden_layers", int), ("hidden_size", int),
                          ("num_attention_heads", int), ("num_key_value_heads", int),
                          ("head_dim", int), ("intermediate_size", int), ("vocab_size", int),
                          ("rope_theta", float), ("rms_norm_eps", float)):
            m = re.search(key + r"=([0-9.e+-]+)", text)
            if m:
                cfg[key] = cast(float(m.group(1)))
        m = re.search(r"tie_word_embeddings=(true|false)", text)
        if m:
            cfg["tie_word_embeddings"] = m.group(1) == "true"
    except (OSError, KeyError, IndexError, ValueError):
        pass
    cfg["architectures"] = ["Qwen3ForCausalLM"]
    return cfg


def benchmark_config():
    """The default shape."""
    return shape_config("4b")


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            raw = json.load(f)
        out = {"hbm_gbs": float(raw["hbm_gbs"]), "bf16_tflops": float(raw["bf16_tflops"]),
               "source": "measured"}
        if "bf16_tflops_sustained" in raw:
            out["bf16_tflops_sustained"] = float(raw["bf16_tflops_sustained"])
        return out
    except (OSError, KeyError, ValueError, TypeError):
        return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """nvidia-smi clocks and throttle reasons while a timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples, self.proc, self.thread = [], None, None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            return
        self.thread = threading.Thread(target=self._read, daemon=True)
        self.thread.start()
        time.sleep(0.3)

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append(line.strip())

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        mhz, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for s in self.samples:
            parts = [p.strip() for p in s.split(",")]
            if len(parts) < 6:
                continue
            try:
                mhz.append(float(parts[0]))
                mx = float(parts[1])
            except ValueError:
                continue
            for n, v in zip(names, parts[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(mhz) if mhz else None, "sm_max_mhz": mx,
                "reasons": sorted(reasons), "samples": len(mhz)}


def make_prompts(shape: str, batch: int, vocab: int, seed: int = 0):
    """Uniform random token ids; equal lengths, or seeded uniform lengths for a (low, high) pair."""
    import torch
    _, _, work = SHAPES[shape]
    g = torch.Generator().manual_seed(seed)
    spec = work["prompt"]
    if isinstance(spec, tuple):
        lengths = torch.randint(spec[0], spec[1] + 1, (batch,), generator=g).tolist()
    else:
        lengths = [spec] * batch
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]


def e2e_new_tokens(steps, context, prompts):
    """New tokens of an end-to-end call, the same for both arms: the timed step count, but no
    fewer than 128 (the longest of the reference's own workloads, bench/bench.py:18-22)."""
    return max(2, min(max(steps, 128), context - max(len(p) for p in prompts)))


def measure_entry(slot, prompt):
    from enginekernel_b200.engine.runner import StepEntry
    return StepEntry(slot, prompt[:PREFILL_TOKENS], [min(len(prompt), PREFILL_TOKENS) - 1])


def timed_generate(engine, prompts, n_new):
    """One whole ``generate`` call on the host's clock: (seconds, seconds to the first token)."""
    import torch
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    first = None
    for _ in engine.generate(prompts, n_new):
        if first is None:
            first = time.perf_counter()
    torch.cuda.synchronize()
    return time.perf_counter() - t0, first - t0


def end_to_end(engine, prompts, n_new, batch):
    """Whole calls until a second has been timed (three at least); medians."""
    list(engine.generate(prompts, n_new))                              # the shape's graphs exist
    calls, total = [], 0.0
    while len(calls) < 3 or (total < MIN_TIMED_SECONDS and len(calls) < 20):
        whole, ttft = timed_generate(engine, prompts, n_new)
        calls.append((whole, ttft))
        total += whole
    whole = statistics.median(c[0] for c in calls)
    ttft = statistics.median(c[1] for c in calls)
    after_first = statistics.median((c[0] - c[1]) for c in calls)
    return {"value": batch * n_new / whole, "unit": "tok/s", "what": "whole generate() calls: "
            "prompt step and every decode step, host lists in, every step read back",
            "new_tokens": n_new, "calls": len(calls), "call_ms": whole * 1e3, "ttft_ms": ttft * 1e3,
            "after_first_token": batch * (n_new - 1) / after_first if n_new > 1 else None,
            "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 4 * batch,
            "prefill_h2d_bytes": 4 * (3 * sum(len(p) for p in prompts) + 2 * batch + 1)}


# --------------------------------------------------------------------------- the reference arm
def run_reference(args) -> int:
    def unavailable(why):
        print(json.dumps({"impl": "reference", "unavailable": why}))
        return 0

    ref_engine = os.path.join(ROOT, "baseline", "_ref", "engine")
    if not os.path.isfile(os.path.join(ref_engine, "engine.py")):
        return unavailable("baseline/_ref holds no copy of the reference tree (engine/engine.py is missing)")
    if args.gpus != 1:
        return unavailable("the reference runs on one GPU only")
    import torch
    if not torch.cuda.is_available():
        return unavailable("no CUDA device here; the reference arm is timed on a GPU only")
    from enginekernel_b200.config import Qwen3Config
    from enginekernel_b200.weights.random_init import write_random_model

    _, _, work = SHAPES[args.shape]
    raw = shape_config(args.shape)
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = Qwen3Config.from_dict(raw)
    batch = args.batch or work["batch"]
    steps = args.steps or work["steps"]
    folder = tempfile.mkdtemp(prefix="ek_ref_model_")
    try:
        write_random_model(folder, cfg, seed=0, device="cuda")
        torch.cuda.empty_cache()
        sys.path.insert(0, ref_engine)
        import engine as reference_engine               # the reference's engine/engine.py, unmodified
        eng = reference_engine.Engine(folder)
        prompts = make_prompts(args.shape, batch, cfg.vocab_size)
        n_new = e2e_new_tokens(steps, work["context"], prompts)
        list(eng.generate(prompts, n_new))                # its graphs for this shape are captured here
        for _ in range(max(0, min(args.warmup, 3) - 1)):
            list(eng.generate(prompts, n_new))
        sampler = ClockSampler()
        sampler.start()
        calls, total = [], 0.0
        while len(calls) < 3 or (total < MIN_TIMED_SECONDS and len(calls) < 20):
            whole, ttft = timed_generate(eng, prompts, n_new)
            calls.append((whole, ttft))
            total += whole
        clocks = sampler.stop()
        whole = statistics.median(c[0] for c in calls)
        ttft = statistics.median(c[1] for c in calls)
        after = statistics.median(c[0] - c[1] for c in calls)
        ms_step = after / (n_new - 1) * 1e3
        out = {
            "impl": "reference",
            "metric": f"decode tok/s ({work['name']} shape, batch {batch})",
            "value": batch / (ms_step / 1e3), "unit": "tok/s", "n_gpus": 1, "steps": n_new - 1,
            "warmup": args.warmup, "ms_per_step": ms_step, "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic: seeded random weights and uniform random token ids",
            "timing": "host clock between the first token and the end of generate(), device "
                      "synchronised (the reference exposes no device-timed step)",
            "config": {"model": f"{work['name']} shape (Qwen3ForCausalLM)", "shape": args.shape,
                       "num_hidden_layers": full_layers, "layers_run": cfg.num_hidden_layers,
                       "hidden_size": cfg.hidden_size, "vocab_size": cfg.vocab_size,
                       "global_batch": batch, "seq_len": work["context"],
                       "prompt_tokens": sum(len(p) for p in prompts), "parallelism": "none (1 GPU)"},
            "clocks": clocks,
            "e2e": {"value": batch * n_new / whole, "unit": "tok/s", "new_tokens": n_new,
                    "calls": len(calls), "call_ms": whole * 1e3, "ttft_ms": ttft * 1e3,
                    "after_first_token": batch * (n_new - 1) / after},
            "reference": {"tier": getattr(eng, "tier", None),
                          "triton": bool(getattr(eng, "triton", False)) if eng.tier == "fast" else False,
                          "graphs": len(getattr(eng, "graphs", {})) if eng.tier == "fast" else 0,
                          "torch": torch.__version__},
        }
        print(json.dumps(out))
        return 0
    finally:
        shutil.rmtree(folder, ignore_errors=True)


# --------------------------------------------------------------------------- two designs side by side
# Layer sizes of real models (width, query heads, key heads, head size, feed-forward width); the
# vocabulary is the Qwen3 one.  Both designs get the same sizes, layer count and workload.
DESIGN_SIZES = {
    "0.6b": dict(width=1024, heads=16, kv_heads=8, dim=128, ff=3072, vocab=151936),
    "4b": dict(width=2560, heads=32, kv_heads=8, dim=128, ff=9728, vocab=151936),
    "1b-h64": dict(width=2048, heads=32, kv_heads=8, dim=64, ff=8192, vocab=128256),
}


def design_configs(size: dict, layers: int, context: int):
    """(Lopazen configuration, Qwen3 configuration) of one size."""
    from enginekernel_b200.config import Qwen3Config
    from enginekernel_b200.config.lopazen import LopazenConfig
    layer = {"type": "attention",
             "mixer": {"dim": size["dim"], "vdim": size["dim"], "heads": size["heads"],
                       "kv_heads": size["kv_heads"], "scale": size["dim"] ** -0.5,
                       "q_temp": {"coef": 0.5, "every": 128}},
             "mlp": {"kind": "dense", "ff": size["ff"]}}
    lopazen = LopazenConfig.from_dict({
        "architecture": "Lopazen", "vocab": size["vocab"], "width": size["width"],
        "embedding": {"scale": size["width"] ** 0.5}, "norm": {"eps": 1e-6}, "layers": [layer] * layers})
    qwen3 = Qwen3Config.from_dict({
        "architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": layers, "hidden_size": size["width"],
        "num_attention_heads": size["heads"], "num_key_value_heads": size["kv_heads"],
        "head_dim": size["dim"], "intermediate_size": size["ff"], "vocab_size": size["vocab"],
        "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": True,
        "max_position_embeddings": context})
    return lopazen, qwen3


# Susalorn at sizes that resemble real layers, each beside a Qwen3 decoder of the same width whose dense
# feed-forward does the work of the experts a token is sent to (ff = top * expert ff * 2 / 3: a gated
# feed-forward has three matrices where an expert has two).  The cached row of the latent attention
# (kv_rank + rot_dim) is 256 values, the most the attention kernels take.
SUSALORN_SIZES = {
    "1b": dict(width=2048, vocab=128256,
               latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=192),
               delta=dict(heads=16, kv_heads=16, dim=128, vdim=128, conv=4, rank=64),
               moe=dict(experts=32, ff=1024, top=4, groups=(4, 2)),
               qwen3=dict(heads=16, kv_heads=8, dim=128, ff=2816)),
    "2b-dense": dict(width=2560, vocab=151936,
                     latent=dict(heads=20, dim=128, rot_dim=64, vdim=128, q_rank=1024, kv_rank=192),
                     delta=dict(heads=20, kv_heads=10, dim=128, vdim=128, conv=4, rank=80),
                     dense=6912, qwen3=dict(heads=20, kv_heads=10, dim=128, ff=6912)),
}


def susalorn_configs(size: dict, layers: int, context: int):
    """(Susalorn configuration, Qwen3 configuration) of one size: latent-attention and delta-rule layers
    in turn, every one with the size's feed-forward, four residual streams."""
    from enginekernel_b200.config import Qwen3Config, SusalornConfig
    la, de = size["latent"], size["delta"]
    if "moe" in size:
        m = size["moe"]
        mlp = {"kind": "moe", "expert": {"ff": m["ff"]},
               "router": {"experts": m["experts"], "top": m["top"], "scale": 2.5,
                          "groups": {"count": m["groups"][0], "keep": m["groups"][1]}}}
    else:
        mlp = {"kind": "dense", "ff": size["dense"]}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": dict(la, scale=(la["dim"] + la["rot_dim"]) ** -0.5,
                            rot={"base": 10000.0, "dims": la["rot_dim"],
                                 "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}})}
    delta = {"type": "channel_delta", "mlp": mlp, "mixer": dict(de)}
    susalorn = SusalornConfig.from_dict({
        "architecture": "Susalorn", "vocab": size["vocab"], "width": size["width"], "norm": {"eps": 1e-6},
        "streams": 4, "layers": [delta if i % 2 == 0 else latent for i in range(layers)]})
    q = size["qwen3"]
    qwen3 = Qwen3Config.from_dict({
        "architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": layers, "hidden_size": size["width"],
        "num_attention_heads": q["heads"], "num_key_value_heads": q["kv_heads"], "head_dim": q["dim"],
        "intermediate_size": q["ff"], "vocab_size": size["vocab"], "rope_theta": 1000000.0,
        "rms_norm_eps": 1e-6, "tie_word_embeddings": True, "max_position_embeddings": context})
    return susalorn, qwen3


# Bolelix at sizes that resemble real layers, beside the Susalorn decoder - the closest design here: it too has
# a recurrent mixer over a per-sequence state, attention layers and routed experts - at the same width, layer
# count, head sizes and experts.  Layers in turn: state-space, attention with a window and kept first tokens,
# matrix memory, attention reading the keys of the attention layer before it.
BOLELIX_SIZES = {
    "1b": dict(width=2048, vocab=128256,
               attention=dict(heads=16, kv_heads=8, dim=128, vdim=128, rot=64, window=1024, keep_first=4),
               mamba2=dict(heads=32, vdim=128, state=128, groups=8, conv=4, norm_groups=8),
               mlstm=dict(heads=16, dim=128, vdim=128, gate_cap=15.0),
               moe=dict(experts=32, ff=1024, top=4), beside=dict(SUSALORN_SIZES["1b"])),
    "2b": dict(width=2560, vocab=151936,
               attention=dict(heads=20, kv_heads=10, dim=128, vdim=128, rot=128, window=512, keep_first=64),
               mamba2=dict(heads=40, vdim=128, state=128, groups=4, conv=4, norm_groups=1),
               mlstm=dict(heads=20, dim=128, vdim=128, gate_cap=15.0),
               moe=dict(experts=16, ff=1536, top=2),
               beside=dict(width=2560, vocab=151936,
                           latent=dict(heads=20, dim=128, rot_dim=64, vdim=128, q_rank=1024, kv_rank=192),
                           delta=dict(heads=20, kv_heads=10, dim=128, vdim=128, conv=4, rank=80),
                           moe=dict(experts=16, ff=1536, top=2, groups=(4, 2)),
                           qwen3=dict(heads=20, kv_heads=10, dim=128, ff=2048))),
}


def bolelix_configs(size: dict, layers: int, context: int):
    """(Bolelix configuration, Susalorn configuration) of one size."""
    from enginekernel_b200.config import BolelixConfig
    at, m = size["attention"], size["moe"]
    mlp = {"kind": "moe", "expert": {"ff": m["ff"]}, "router": {"experts": m["experts"], "top": m["top"]}}
    attn = {"dim": at["dim"], "vdim": at["vdim"], "heads": at["heads"], "kv_heads": at["kv_heads"],
            "scale": at["dim"] ** -0.5 * 8.0, "rot": {"base": 1000000.0, "dims": at["rot"], "scaling": {"factor": 4.0}},
            "mask": {"size": at["window"], "keep_first": at["keep_first"]}}
    made = []
    for i in range(layers):
        kind = i % 4
        if kind == 0:
            made.append({"type": "mamba2", "mixer": dict(size["mamba2"]), "mlp": mlp})
        elif kind == 2:
            made.append({"type": "mlstm", "mixer": dict(size["mlstm"]), "mlp": mlp})
        else:
            made.append({"type": "attention", "mixer": dict(attn, **({"kv_from": i - 2} if kind == 3 else {})), "mlp": mlp})
    bolelix = BolelixConfig.from_dict({"architecture": "Bolelix", "vocab": size["vocab"], "width": size["width"],
                                       "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "layers": made})
    return bolelix, susalorn_configs(size["beside"], layers, context)[0]


# Musavik at sizes that resemble real layers, beside the Bolelix decoder - the closest design here: it too has
# attention behind a window that keeps the first tokens, with a gate on its result, in turn with recurrences behind a
# short convolution - at the same width, layer count and head sizes.  Layers in turn: recurrence, recurrence, the
# pair of attention and delta rule; the whole stack is one pass of a loop, so that the input mix runs once a step.
MUSAVIK_SIZES = {
    "1b": dict(width=2048, vocab=128256, rglru=dict(width=2048, blocks=8, conv=4),
               left=dict(heads=16, kv_heads=4, dim=128, vdim=128, rot=64, window=1024, keep_first=4),
               right=dict(heads=16, kv_heads=8, dim=128, vdim=128, conv=4), ff=6144, pairs=(99991, 127, 17),
               beside="1b"),
    "2b": dict(width=2560, vocab=151936, rglru=dict(width=2560, blocks=10, conv=4),
               left=dict(heads=20, kv_heads=5, dim=128, vdim=128, rot=128, window=512, keep_first=64),
               right=dict(heads=20, kv_heads=10, dim=128, vdim=128, conv=4), ff=7680, pairs=(199999, 8191, 31),
               beside="2b"),
}


def musavik_configs(size: dict, layers: int, context: int):
    """(Musavik configuration, Bolelix configuration) of one size."""
    from enginekernel_b200.config.musavik import MusavikConfig
    at = size["left"]
    left = {"dim": at["dim"], "vdim": at["vdim"], "heads": at["heads"], "kv_heads": at["kv_heads"],
            "scale": at["dim"] ** -0.5 * 8.0, "rot": {"base": 1000000.0, "dims": at["rot"]},
            "mask": {"size": at["window"], "keep_first": at["keep_first"]}}
    mlp = {"kind": "dense", "ff": size["ff"]}
    made = []
    for i in range(layers):
        if i % 3 == 2:
            made.append({"type": "parallel", "mlp": mlp,
                         "mixer": {"left": left, "right": dict(size["right"]), "left_scale": 0.8, "right_scale": 0.5}})
        else:
            made.append({"type": "rglru", "mixer": dict(size["rglru"]), "mlp": mlp})
    b, mp, mc = size["pairs"]
    musavik = MusavikConfig.from_dict({
        "architecture": "Musavik", "vocab": size["vocab"], "width": size["width"], "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.0, "bigram": {"buckets": b, "mul_prev": mp, "mul_cur": mc}}, "layers": made,
        "loop": {"start": 0, "stop": layers, "times": 1}})
    return musavik, bolelix_configs(BOLELIX_SIZES[size["beside"]], layers, context)[0]


# Kamosun at sizes that resemble real layers, beside the Bolelix decoder - the closest design here: it too runs both
# sublayers of a layer side by side on the same stream, mixes attention (with keys shared between layers) with
# recurrences over the decay scan, and has gated experts - at the same width, layer count, head sizes and experts.
# Layers in turn: the pair of full attention and fixed-decay memory, chunked attention, chunked attention that reads
# the keys of the layer before it, chunked attention; the first layer's feed-forward is dense.
KAMOSUN_SIZES = {
    "1b": dict(width=2048, vocab=128256,
               left=dict(heads=16, kv_heads=8, dim=128, vdim=128, rot=128), right=dict(heads=16, dim=128, vdim=128),
               attention=dict(heads=16, kv_heads=8, dim=128, vdim=128, rot=128, chunk=1024),
               moe=dict(experts=32, ff=1024, top=4, shared=1024), dense=6144, beside="1b"),
    "2b": dict(width=2560, vocab=151936,
               left=dict(heads=10, kv_heads=10, dim=128, vdim=256, rot=128), right=dict(heads=20, dim=128, vdim=128),
               attention=dict(heads=20, kv_heads=10, dim=128, vdim=128, rot=64, chunk=512),
               moe=dict(experts=16, ff=1536, top=2, shared=2048), dense=7680, beside="2b"),
}


def kamosun_configs(size: dict, layers: int, context: int):
    """(Kamosun configuration, Bolelix configuration) of one size."""
    from enginekernel_b200.config.kamosun import KamosunConfig

    def attention(at, **more):
        return dict({"dim": at["dim"], "vdim": at["vdim"], "heads": at["heads"], "kv_heads": at["kv_heads"],
                     "scale": at["dim"] ** -0.5, "rot": {"base": 1000000.0, "dims": at["rot"]}}, **more)

    at, right, m = size["attention"], size["right"], size["moe"]
    left = attention(size["left"], softcap=30.0)
    left["rot"]["scaling"] = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}
    decay = [math.exp(-2.0 ** (-8.0 * (h + 1) / right["heads"])) for h in range(right["heads"])]
    moe = {"kind": "moe", "expert": {"ff": m["ff"], "limit": 7.0}, "shared": {"ff": m["shared"], "limit": 7.0},
           "router": {"experts": m["experts"], "top": m["top"]}}
    made = []
    for i in range(layers):
        if i % 4 == 0:
            mixer = {"left": left, "right": dict(right, decay=decay)}
        else:
            mixer = attention(at, mask={"size": at["chunk"]}, **({"kv_from": i - 1} if i % 4 == 2 else {}))
        made.append({"type": "attention" if i % 4 else "parallel", "mixer": mixer,
                     "mlp": moe if i else {"kind": "dense", "ff": size["dense"], "limit": 7.0}})
    kamosun = KamosunConfig.from_dict({"architecture": "Kamosun", "vocab": size["vocab"], "width": size["width"],
                                       "norm": {"eps": 1e-6}, "residual_mult": 0.5, "layers": made})
    return kamosun, bolelix_configs(BOLELIX_SIZES[size["beside"]], layers, context)[0]


# Gesuvik at sizes that resemble real layers, beside the Kamosun decoder - the closest design here: it too mixes
# attention over a part of the context with linear attention over the decay scan, and has clamped gated experts beside a
# shared one - at the same width, layer count, head sizes and experts.  Layers in turn: retention, latent attention,
# retention, attention.
GESUVIK_SIZES = {
    "1b": dict(width=2048, vocab=128256, retention=dict(heads=16, dim=128, vdim=128),
               latent=dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=192, window=1024),
               attention=dict(heads=16, kv_heads=8, dim=128, vdim=128, rot=128, window=1024),
               moe=dict(experts=32, identity=8, ff=1024, top=4, shared=1024), beside="1b"),
    "2b": dict(width=2560, vocab=151936, retention=dict(heads=10, dim=256, vdim=256),
               latent=dict(heads=20, dim=128, rot_dim=64, vdim=192, kv_rank=160, window=512),
               attention=dict(heads=20, kv_heads=10, dim=128, vdim=128, rot=64, window=512),
               moe=dict(experts=16, identity=4, ff=1536, top=2, shared=2048), beside="2b"),
}


def gesuvik_configs(size: dict, layers: int, context: int):
    """(Gesuvik configuration, Kamosun configuration) of one size."""
    from enginekernel_b200.config.gesuvik import GesuvikConfig
    at, la, re_, m = size["attention"], size["latent"], size["retention"], size["moe"]
    moe = {"kind": "moe", "expert": {"ff": m["ff"], "limit": 7.0}, "shared": {"ff": m["shared"], "limit": 7.0},
           "router": {"experts": m["experts"], "identity": m["identity"], "top": m["top"]}}
    attention = {"dim": at["dim"], "vdim": at["vdim"], "heads": at["heads"], "kv_heads": at["kv_heads"],
                 "scale": at["dim"] ** -0.5, "mask": {"size": at["window"]},
                 "rot": {"base": 1000000.0, "dims": at["rot"],
                         "scaling": {"factor": 4.0, "fast": 32.0, "original": 8192, "slow": 1.0}}}
    latent = {"heads": la["heads"], "dim": la["dim"], "rot_dim": la["rot_dim"], "vdim": la["vdim"],
              "kv_rank": la["kv_rank"], "scale": (la["dim"] + la["rot_dim"]) ** -0.5, "mask": {"size": la["window"]},
              "rot": {"base": 1000000.0, "dims": la["rot_dim"]}}
    retention = dict(re_, decay=[1.0 - 2.0 ** (-5.0 - 6.0 * h / re_["heads"]) for h in range(re_["heads"])],
                     rot={"base": 10000.0, "dims": re_["dim"]})
    turn = [("retention", retention), ("latent_attention", latent), ("retention", retention), ("attention", attention)]
    made = [{"type": turn[i % 4][0], "mixer": turn[i % 4][1], "mlp": moe} for i in range(layers)]
    gesuvik = GesuvikConfig.from_dict({"architecture": "Gesuvik", "vocab": size["vocab"], "width": size["width"],
                                       "norm": {"eps": 1e-6}, "logit_scale": 0.5, "logit_softcap": 30.0, "layers": made})
    return gesuvik, kamosun_configs(KAMOSUN_SIZES[size["beside"]], layers, context)[0]


#: design -> (sizes, configurations of one size, the design it is measured beside)
DESIGNS = {"lopazen": (DESIGN_SIZES, design_configs, "qwen3"), "susalorn": (SUSALORN_SIZES, susalorn_configs, "qwen3"),
           "bolelix": (BOLELIX_SIZES, bolelix_configs, "susalorn"), "musavik": (MUSAVIK_SIZES, musavik_configs, "bolelix"),
           "kamosun": (KAMOSUN_SIZES, kamosun_configs, "bolelix"), "gesuvik": (GESUVIK_SIZES, gesuvik_configs, "kamosun")}


def measure_design(cfg, vocab, batch, prompt_len, context, steps, warmup, pk, with_kernels):
    """Prompt step and decode step of one model: milliseconds, tokens a second, per-kernel tables."""
    import torch
    from enginekernel_b200 import Engine, SamplingParams, measure
    from enginekernel_b200.engine.runner import StepEntry
    engine = Engine.from_config(cfg, seed=0, dtype="bfloat16", max_tokens=batch * context, max_batch=batch,
                                max_len=context)
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, vocab, (prompt_len,), generator=g).tolist() for _ in range(batch)]
    times = []
    for it in range(3 + 5):
        slot = engine.open_sequence()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        engine.step([(slot, prompts[0], [prompt_len - 1])])
        b.record()
        torch.cuda.synchronize()
        engine.close_sequence(slot)
        if it >= 3:
            times.append(a.elapsed_time(b))
    out = {"prefill_ms": statistics.median(times)}
    out["prefill_tok_s"] = prompt_len / (out["prefill_ms"] / 1e3)
    room = context - prompt_len - 8
    run = engine.backend.start(prompts, [room] * batch, SamplingParams(), [], list(range(batch)))
    try:
        st = run.state
        for _ in range(warmup):
            st.step()
        torch.cuda.synchronize()
        stretches = 5                                # median of five stretches of k steps
        k = max(1, min(steps, (room - warmup - 40) // stretches))
        per_step = []
        for _ in range(stretches):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            for _ in range(k):
                st.step()
            b.record()
            torch.cuda.synchronize()
            per_step.append(a.elapsed_time(b) / k)
        out["decode_ms"] = statistics.median(per_step)
        out["decode_ms_spread"] = [min(per_step), max(per_step)]
        out["decode_tok_s"] = batch / (out["decode_ms"] / 1e3)
        out["decode_steps"], out["launches_per_step"] = k, st.launches_per_step
        weight_bytes = engine.model.weight_bytes_read_per_step()
        live = prompt_len + warmup + stretches * k // 2
        kv = 0                                       # what a step reads of the cache: pages, or a state both ways
        for cs in engine.model.cache_entry_specs():
            if cs is not None and cs.kind == "kv":
                kv += cs.planes * 2 * batch * live * cs.heads * cs.head_dim
            elif cs is not None:
                size = 1
                for d in cs.shape:
                    size *= d
                kv += 2 * 4 * batch * size
        out["decode_frac_of_copy_bandwidth"] = (weight_bytes + kv) / (out["decode_ms"] / 1e3) / 1e9 / pk["hbm_gbs"]
        if with_kernels:
            out["decode_kernels"] = measure.decode_step_table(st, pk)
    finally:
        run.close()
    if with_kernels:
        slot = engine.open_sequence()
        try:
            out["prefill_kernels"] = measure.prefill_step_table(
                lambda: engine.runner.step([StepEntry(slot, prompts[0], [prompt_len - 1])]), pk)
        finally:
            engine.close_sequence(slot)
    del engine
    torch.cuda.empty_cache()
    return out


def run_designs(args) -> int:
    """``--design NAME``: that decoder beside the Qwen3 decoder at equal layer sizes."""
    import torch
    if not torch.cuda.is_available():
        print(json.dumps({"design": args.design, "unavailable": "no CUDA device here"}))
        return 0
    pk = peaks()
    layers = args.layers or 12
    batch = args.batch or 8
    prompt_len, context = PREFILL_TOKENS, 4096
    steps = args.steps or 128
    sampler = ClockSampler()
    sampler.start()
    sizes = {}
    design_sizes, make_configs, beside = DESIGNS[args.design]
    for name in (args.sizes.split(",") if args.sizes else list(design_sizes)):
        size = design_sizes[name]
        design, other = make_configs(size, layers, context)
        sizes[name] = {"size": size, "layers": layers}
        for tag, cfg in ((args.design, design), (beside, other)):
            sizes[name][tag] = measure_design(cfg, size["vocab"], batch, prompt_len, context, steps,
                                              max(3, args.warmup), pk, not args.skip_kernels)
        a, b = sizes[name][args.design], sizes[name][beside]
        sizes[name][f"{args.design}_over_{beside}"] = {"prefill_tok_s": a["prefill_tok_s"] / b["prefill_tok_s"],
                                                       "decode_tok_s": a["decode_tok_s"] / b["decode_tok_s"]}
    print(json.dumps({
        "design": args.design, "beside": beside, "dtype": "bf16", "n_gpus": 1,
        "data": "synthetic: seeded random weights and uniform random token ids",
        "workload": {"batch": batch, "prompt_tokens": prompt_len, "context": context, "decode_steps": f"median of 5 stretches of {steps}",
                     "prefill": "one prompt of 2,048 tokens in one step", "timing": "CUDA events",
                     "l2": "step inputs (weights and cache of all layers) exceed the 126 MB L2"},
        "peaks": pk, "clocks": sampler.stop(), "sizes": sizes}))
    return 0


# --------------------------------------------------------------------------- this repository's arm
def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=0, help="decode steps timed at a stretch (default: the shape's)")
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--shape", default="4b", choices=sorted(SHAPES))
    ap.add_argument("--layers", type=int, default=0,
                    help="run fewer layers than the configuration has (both numbers are reported)")
    ap.add_argument("--batch", type=int, default=0, help="sequences in the batch (default: the shape's)")
    ap.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64")
    ap.add_argument("--skip-kernels", action="store_true", help="leave out the per-kernel tables")
    ap.add_argument("--prefill-seqs", type=int, default=1,
                    help="sequences of 2,048 tokens in the prompt step of the per-kernel table")
    ap.add_argument("--design", default="", choices=["", "lopazen", "susalorn", "bolelix", "musavik", "kamosun", "gesuvik"],
                    help="instead of the default workload: this design beside the Qwen3 decoder (bolelix: beside "
                         "the Susalorn decoder; musavik, kamosun: beside the Bolelix decoder; gesuvik: beside the Kamosun decoder) at equal layer sizes (prompt "
                         "step, decode step, per-kernel tables)")
    ap.add_argument("--sizes", default="", help="with --design: comma-separated names of DESIGN_SIZES")
    args = ap.parse_args(argv)

    if args.design:
        return run_designs(args)
    if args.impl == "reference":
        return run_reference(args)
    if args.gpus != 1:
        print(f"bench.py measures one GPU only (this library runs on a single B200); --gpus {args.gpus} is not run")
        return 2
    warmup = max(3, args.warmup)

    import torch
    from enginekernel_b200 import Engine, SamplingParams, measure
    from enginekernel_b200.config import Qwen3Config
    from enginekernel_b200.ops.lib import loaded_libraries
    from enginekernel_b200.engine.runner import DEFAULT_MAX_STEP_TOKENS

    _, _, work = SHAPES[args.shape]
    raw = shape_config(args.shape)
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = Qwen3Config.from_dict(raw)
    pk = peaks()
    batch = args.batch or work["batch"]
    steps = args.steps or work["steps"]
    context = work["context"]
    with_points = args.shape == "4b" and not args.skip_points
    biggest = max(batch, 64 if with_points else 1)
    engine = Engine.from_config(cfg, seed=0, dtype="bfloat16", max_tokens=biggest * context,
                                max_batch=biggest, max_len=context,
                                max_step_tokens=max(DEFAULT_MAX_STEP_TOKENS, args.prefill_seqs * PREFILL_TOKENS))
    L, H, NH, NKV, D, I, V = (cfg.num_hidden_layers, cfg.hidden_size, cfg.num_attention_heads,
                              cfg.num_key_value_heads, cfg.head_dim, cfg.intermediate_size,
                              cfg.vocab_size)
    kv_per_token = 2 * L * NKV * D * 2
    weight_bytes = engine.model.weight_bytes_read_per_step()

    # ---- prefill of 2,048 tokens -------------------------------------------------------
    one = make_prompts("4b", 1, V, seed=1)[0][:PREFILL_TOKENS]
    times = []
    for it in range(4 + 5):                      # 4 warm-ups (clocks, workspace), median of 5
        slot = engine.open_sequence()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        engine.step([(slot, one, [PREFILL_TOKENS - 1])])
        b.record()
        torch.cuda.synchronize()
        engine.close_sequence(slot)
        if it >= 4:
            times.append(a.elapsed_time(b))
    prefill_ms = statistics.median(times)
    per_token_linear = 2 * L * (H * (NH + 2 * NKV) * D + NH * D * H + 3 * H * I)
    attn_flops = L * 4 * NH * D * PREFILL_TOKENS * (PREFILL_TOKENS + 1) / 2
    prefill_flops = per_token_linear * PREFILL_TOKENS + attn_flops + 2 * H * V
    prefill = {"value": PREFILL_TOKENS / (prefill_ms / 1e3), "tokens": PREFILL_TOKENS, "ms": prefill_ms,
               "frac": prefill_flops / (prefill_ms / 1e3) / (pk["bf16_tflops"] * 1e12)}

    # ---- decode --------------------------------------------------------------------------
    def decode(b, k, sample_clocks=False, kernels=False):
        """K steps at a stretch, repeated until a second has been timed (or the context is full)."""
        prompts = make_prompts(args.shape, b, V)
        longest = max(len(p) for p in prompts)
        slack = 32                                # steps the per-kernel measurement replays
        room = min(context - longest - warmup - slack, STEP_BUDGET)
        k = max(1, min(k, room))
        run = engine.backend.start(prompts, [warmup + room + slack] * b, SamplingParams(), [],
                                   list(range(b)))
        try:
            st = run.state
            for _ in range(warmup):
                st.step()
            torch.cuda.synchronize()
            sampler = ClockSampler() if sample_clocks else None
            if sampler:
                sampler.start()
            total_ms, repeats, done = 0.0, 0, warmup
            while repeats == 0 or (total_ms < MIN_TIMED_SECONDS * 1e3 and done + k <= room + warmup):
                a, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                for _ in range(k):
                    st.step()
                e.record()
                torch.cuda.synchronize()
                total_ms += a.elapsed_time(e)
                repeats += 1
                done += k
            clocks = sampler.stop() if sampler else None
            ms = total_ms / (repeats * k)
            mean_context = sum(len(p) for p in prompts) / b + warmup + (done - warmup) / 2
            table = None
            if kernels:
                table = measure.decode_step_table(st, pk)
                table["batch"], table["context"] = b, int(mean_context + (done - warmup) / 2)
            return {"ms": ms, "clocks": clocks, "launches": st.launches_per_step, "repeats": repeats,
                    "steps": k, "mean_context": mean_context, "kernels": table}
        finally:
            run.close()

    main_run = decode(batch, steps, sample_clocks=True, kernels=not args.skip_kernels)
    ms_step = main_run["ms"]
    value = batch / (ms_step / 1e3)
    step_bytes = weight_bytes + batch * main_run["mean_context"] * kv_per_token
    achieved = step_bytes / (ms_step / 1e3) / 1e9
    roofline = {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s",
                "frac": achieved / pk["hbm_gbs"], "peaks": pk["source"]}

    points, point_fracs = {}, {}
    if with_points:
        for b in (1, 64):
            r = decode(b, max(16, steps // 2))
            points[f"decode_b{b}"] = b / (r["ms"] / 1e3)
            bytes_b = weight_bytes + b * r["mean_context"] * kv_per_token
            point_fracs[f"decode_b{b}"] = bytes_b / (r["ms"] / 1e3) / 1e9 / pk["hbm_gbs"]

    kernels = {}
    if main_run["kernels"] is not None:
        kernels["decode"] = main_run["kernels"]
        n_pre = max(1, min(args.prefill_seqs, biggest))
        many = make_prompts("4b", n_pre, V, seed=1)
        slots = [engine.open_sequence() for _ in many]
        try:
            kernels["prefill"] = measure.prefill_step_table(
                lambda: engine.runner.step([measure_entry(s, p) for s, p in zip(slots, many)]), pk)
            kernels["prefill"]["tokens"] = n_pre * PREFILL_TOKENS
        finally:
            for s in slots:
                engine.close_sequence(s)

    # ---- end to end through Engine.generate --------------------------------------------
    host_prompts = make_prompts(args.shape, batch, V)
    n_new = e2e_new_tokens(steps, context, host_prompts)
    e2e = end_to_end(engine, host_prompts, n_new, batch)

    prompt_desc = work["prompt"]
    out = {
        "metric": f"decode tok/s ({work['name']} shape, batch {batch}, "
                  + (f"{prompt_desc[0]}-{prompt_desc[1]}-token prompts)" if isinstance(prompt_desc, tuple)
                     else f"{prompt_desc:,}-token prompts)"),
        "value": value, "unit": "tok/s", "n_gpus": 1, "steps": main_run["steps"], "warmup": warmup,
        "repeats": main_run["repeats"], "ms_per_step": ms_step, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: seeded random weights and uniform random token ids",
        "config": {
            "model": f"{work['name']} shape (Qwen3ForCausalLM)", "shape": args.shape,
            "num_hidden_layers": full_layers, "layers_run": cfg.num_hidden_layers, "hidden_size": H,
            "num_attention_heads": NH, "num_key_value_heads": NKV, "head_dim": D,
            "intermediate_size": I, "vocab_size": V, "tie_word_embeddings": cfg.tie_word_embeddings,
            "rope_theta": cfg.rope_theta, "global_batch": batch, "seq_len": context,
            "prompt_len": prompt_desc if not isinstance(prompt_desc, tuple) else
            int(sum(len(p) for p in host_prompts) / batch),
            "parallelism": "none (1 GPU)",
            "l2": "step inputs (gigabytes of weights and cache) exceed the 126 MB L2",
            "peaks": pk["source"]},
        "clocks": main_run["clocks"], "e2e": e2e,
        "gpu_launches": main_run["launches"] * main_run["steps"] * main_run["repeats"],
        "prefill": prefill, "roofline": roofline, "points": points, "point_fracs": point_fracs,
        "kernels": kernels,
        "kernel_libraries": sorted(os.path.basename(p) for p in loaded_libraries().values()),
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
