"""Decode and prefill throughput of starter_b200 at Qwen3-4B size on ONE B200, random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

Prints one JSON line.  A "step" is one decode step of the whole batch.  ``value`` is decoded
tokens per second at batch 8, timed on the device with CUDA events around K consecutive steps of
the captured, self-feeding decode step at the middle of the generation range (context 3,072 of
4,096); ``e2e`` is the same through ``Engine.generate``: host ids out every step, the host-owned inputs
of every step in from pinned memory, a step launched before the one before it is read;
``prefill`` is one 2,048-token prompt; ``points`` are decode at batch 1 and 64; ``roofline`` sets the
bytes a decode step must read (every weight it uses once, the live requests' keys and values)
against the measured copy bandwidth.  Every step reads >8 GB of weights, far more than the 126 MB
L2, so nothing is flushed between steps.
"""

from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_4B = dict(
    architectures=["Qwen3ForCausalLM"], num_hidden_layers=36, hidden_size=2560, num_attention_heads=32,
    num_key_value_heads=8, head_dim=128, intermediate_size=9728, vocab_size=151936, rope_theta=5e6,
    rms_norm_eps=1e-6, tie_word_embeddings=True, max_position_embeddings=4096,
)
QWEN3_8B = dict(QWEN3_4B, hidden_size=4096, intermediate_size=12288, rope_theta=1e6, tie_word_embeddings=False)
QWEN3_14B = dict(QWEN3_8B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408)
#: the further rows of the measurement table: model sizes, and the generation workload quoted for each
WORKLOADS = {
    "8b": dict(config=QWEN3_8B, name="Qwen3-8B", batch=8, prompt_range=(512, 2048), new_tokens=256),
    "14b": dict(config=QWEN3_14B, name="Qwen3-14B", batch=32, prompt_range=(1024, 1024), new_tokens=512),
}
CONTEXT = 4096
PROMPT = 2048
DECODE_AT = 3072  # 2,048 prompt tokens + 1,024 decoded: the middle of the generation range


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    out = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}
    if os.path.isfile(path):
        try:
            raw = json.load(open(path))
            out["hbm_gbs"] = float(raw.get("hbm_gbs", out["hbm_gbs"]))
            out["bf16_tflops"] = float(raw.get("bf16_tflops", out["bf16_tflops"]))
            out["bf16_tflops_sustained"] = float(raw.get("bf16_tflops_sustained", out["bf16_tflops_sustained"]))
            out["source"] = "measured"
        except Exception:  # noqa: BLE001
            pass
    return out


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed regions run."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.monotonic(), line.strip()))

    def stop(self, windows):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        clocks, max_clock, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for stamp, line in self.samples:
            if not any(a <= stamp <= b for a, b in windows):
                continue
            parts = [p.strip() for p in line.split(",")]
            try:
                clocks.append(int(parts[0]))
                max_clock = int(parts[1])
            except (ValueError, IndexError):
                continue
            for name, flag in zip(names, parts[2:6]):
                if flag.lower().startswith("active"):
                    reasons.add(name)
        clocks.sort()
        return {"sm_mhz": clocks[len(clocks) // 2] if clocks else None, "sm_max_mhz": max_clock,
                "reasons": sorted(reasons), "samples": len(clocks)}


METRIC = "decode tok/s at batch 8 (Qwen3-4B BF16); prefill tok/s at 2,048 tokens; batch 1/64 in points"


def config_block(layers: int, batch: int, peaks_source: str) -> dict:
    """Every size of the run, flat; the same for both arms."""
    c = QWEN3_4B
    return {
        "model": "Qwen3-4B", "layers": layers, "layers_of_model": c["num_hidden_layers"],
        "hidden": c["hidden_size"], "heads": c["num_attention_heads"], "kv_heads": c["num_key_value_heads"],
        "head_dim": c["head_dim"], "intermediate": c["intermediate_size"], "vocab": c["vocab_size"],
        "tied": True, "global_batch": batch, "seq_len": CONTEXT, "prompt_len": PROMPT,
        "decode_context": DECODE_AT, "parallelism": "single", "l2": "inputs larger than L2",
        "cache_page": 64, "peaks": peaks_source,
    }


def reference_arm(args) -> int:
    """The reference's own engine on the same workload (baseline/reference_arm.py)."""
    from baseline import reference_arm as arm

    sizes = dict(QWEN3_4B, num_hidden_layers=args.layers)
    return arm.run(args, sizes, CONTEXT, PROMPT, DECODE_AT,
                   config_block(args.layers, args.batch, peaks()["source"]), ClockSampler(), METRIC)


def per_stage(model, runner, slots, batch, peak_gbs, out=sys.stderr):
    """Where a decode step's time goes: every kind of kernel of a layer alone, in a CUDA graph that
    runs it once per layer on that layer's own weights and cache (so nothing stays in L2 from one
    launch to the next), timed with CUDA events; against the time its bytes take at the copy peak."""
    import torch

    from starter_b200 import ops

    spec = model.spec
    dev = model.device
    blocks = [model.blocks[e.layer] for e in spec.schedule]
    entries = [e.cache for e in spec.schedule]
    mixer = blocks[0].mixer.spec
    h = spec.hidden_size
    x = (torch.randn(batch, h, device=dev) * 0.5).to(torch.bfloat16)
    res = x.clone()
    attn_in = (torch.randn(batch, mixer.num_heads * mixer.head_dim, device=dev) * 0.5).to(torch.bfloat16)
    act = (torch.randn(batch, blocks[0].feed_forward.down.shape[1], device=dev) * 0.5).to(torch.bfloat16)
    qkv = (torch.randn(batch, blocks[0].mixer.qkv.shape[0], device=dev) * 0.5).to(torch.bfloat16)
    cache = runner.cache
    seq_slot = torch.tensor(slots, dtype=torch.int32, device=dev)
    kv_len = torch.tensor([cache.lengths[s] for s in slots], dtype=torch.int32, device=dev)
    kv_tokens = max(cache.lengths[s] for s in slots)
    rot = blocks[0].mixer.position.rotation()

    def attention(b, entry):
        keys, values = cache.entry_pages(entry)
        m = b.mixer
        return ops.attention_decode_qkv(qkv, keys, values, cache.block_table, seq_slot, kv_len, mixer.num_heads,
                                        mixer.num_kv_heads, mixer.head_dim, mixer.scale, mixer.window, m.q_norm,
                                        m.k_norm, mixer.qk_norm_eps, rot.cos, rot.sin, write_cache=True,
                                        kv_hint=kv_tokens, early=True)

    nbytes = lambda t: t.numel() * t.element_size()
    kv_bytes = cache.bytes_per_token() // len(set(entries)) * int(kv_len.sum())
    stages = [
        ("sum + norm (x2 per layer)", lambda b, e: ops.rmsnorm(res, b.norm1.weight, b.norm1.spec.eps, delta=x), lambda b: 0),
        ("q/k/v projection", lambda b, e: ops.linear(x, b.mixer.qkv), lambda b: nbytes(b.mixer.qkv)),
        ("attention (norm, rotation, cache write inside)", attention, lambda b: kv_bytes),
        ("output projection", lambda b, e: ops.linear(attn_in, b.mixer.o), lambda b: nbytes(b.mixer.o)),
        ("gate/up projection + SwiGLU", lambda b, e: ops.linear(x, b.feed_forward.gate_up, gated=True),
         lambda b: nbytes(b.feed_forward.gate_up)),
        ("down projection", lambda b, e: ops.linear(act, b.feed_forward.down), lambda b: nbytes(b.feed_forward.down)),
    ]
    rows, total = [], 0.0
    for name, fn, bytes_of in stages:
        for b, e in zip(blocks, entries):
            fn(b, e)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for b, e in zip(blocks, entries):
                fn(b, e)
        graph.replay()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        for _ in range(5):
            graph.replay()
        stop.record()
        torch.cuda.synchronize()
        us = start.elapsed_time(stop) / 5 / len(blocks) * 1e3
        ideal = bytes_of(blocks[0]) / (peak_gbs * 1e9) * 1e6
        per_layer = us * (2 if name.startswith("sum") else 1)
        total += per_layer
        rows.append((name, us, ideal))
    print(f"decode step at batch {batch}, {kv_tokens} cached tokens per sequence: microseconds per launch, "
          f"inside a CUDA graph", file=out)
    for name, us, ideal in rows:
        frac = f"{ideal / us:.2f}" if ideal else "-"
        print(f"  {name:48s} {us:7.1f} us   bytes at {peak_gbs:.0f} GB/s: {ideal:6.1f} us   fraction {frac}", file=out)
    print(f"  a layer's seven launches one by one: {total:.1f} us", file=out)
    return total


def workload(args) -> int:
    """One of the further rows (``--workload 8b|14b``): a batch of prompts generated to the end through
    ``Engine.generate``, timed by the wall clock with the device idle on both sides.  Prints one JSON
    line: the whole job's generated tokens a second, the time to the first token (all prompts in one
    step), decode tokens a second after it, and the decode's share of its own memory roofline."""
    import torch

    from starter_b200.config import config_from_dict
    from starter_b200.engine import random_model
    from starter_b200.engine.entry import Engine

    spec = WORKLOADS[args.workload]
    raw = dict(spec["config"])
    layers_of_model = raw["num_hidden_layers"]
    raw["num_hidden_layers"] = min(args.layers, layers_of_model) if args.layers_given else layers_of_model
    config = config_from_dict(raw)
    model = random_model(config, seed=0, dtype="bfloat16")
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    lo, hi = spec["prompt_range"]
    lengths = [int(torch.randint(lo, hi + 1, (1,), generator=gen)) for _ in range(spec["batch"])]
    prompts = [torch.randint(0, config.vocab_size, (n,), generator=gen).tolist() for n in lengths]
    new = spec["new_tokens"]
    engine = Engine.from_model(model, max_batch=spec["batch"])
    sampler = ClockSampler()
    sampler.start()
    for _ in engine.generate(prompts, 4):        # builds the cache, compiles, captures the first graphs
        pass
    best = None
    for _ in range(2):
        torch.cuda.synchronize()
        t0 = time.monotonic()
        stream = engine.generate(prompts, new)
        next(stream)
        torch.cuda.synchronize()
        t1 = time.monotonic()
        for _ in stream:
            pass
        torch.cuda.synchronize()
        t2 = time.monotonic()
        if best is None or t2 - t0 < best[2] - best[0]:
            best = (t0, t1, t2)
    t0, t1, t2 = best
    engine.runner.check_status()
    batch = spec["batch"]
    decode_ms = (t2 - t1) / (new - 1) * 1e3
    mean_context = sum(lengths) / batch + new / 2
    step_bytes = model.step_weight_bytes() + engine.runner.cache.bytes_per_token() * batch * mean_context
    achieved = step_bytes / (decode_ms * 1e-3) / 1e9
    line = {
        "metric": f"generated tok/s of the whole job ({spec['name']} BF16): {batch} prompts of {lo}-{hi} tokens, {new} new tokens each",
        "value": round(batch * new / (t2 - t0), 1), "unit": "tok/s", "n_gpus": 1, "higher_is_better": True,
        "dtype": "bf16", "data": "synthetic: random weights N(0,0.02), uniform random token ids",
        "config": {"model": spec["name"], "layers": raw["num_hidden_layers"], "layers_of_model": layers_of_model,
                   "hidden": raw["hidden_size"], "heads": raw["num_attention_heads"],
                   "kv_heads": raw["num_key_value_heads"], "head_dim": raw["head_dim"],
                   "intermediate": raw["intermediate_size"], "vocab": raw["vocab_size"],
                   "tied": raw["tie_word_embeddings"], "global_batch": batch, "prompt_tokens": sum(lengths),
                   "new_tokens": new, "peaks": pk["source"]},
        "ttft_ms": round((t1 - t0) * 1e3, 2),
        "prefill_tok_s": round(sum(lengths) / (t1 - t0), 1),
        "decode_tok_s": round(batch / decode_ms * 1e3, 1), "decode_ms_per_step": round(decode_ms, 4),
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "clocks": sampler.stop([(t0, t2)]),
    }
    print(json.dumps(line))
    return 0


#: sizes for ``--design goguvik``: layers that resemble a real model's (random weights).  Both designs get
#: the same width, feed-forward, vocabulary, head counts, 128 key columns and 128 value columns per head.
DESIGN_SIZES = {
    "2048": dict(width=2048, ff=8192, heads=16, kv_heads=4, vocab=32768),
    "2560": dict(width=2560, ff=9728, heads=32, kv_heads=8, vocab=151936),
    "4096": dict(width=4096, ff=12288, heads=32, kv_heads=8, vocab=151936),
}


def goguvik_config(size: dict, layers: int) -> dict:
    """Goguvik at ``size``: four streams; of every three layers the second and third attend over the
    keys and values of the first."""
    out = []
    for i in range(layers):
        mixer = dict(heads=size["heads"], kv_heads=size["kv_heads"], dim=64, vdim=128, scale=0.125, diff=0.25,
                     q_temp=dict(coef=0.5, every=128))
        if i % 3:
            mixer["kv_from"] = i - i % 3
        out.append(dict(type="attention", mixer=mixer, mlp=dict(kind="dense", ff=size["ff"])))
    return dict(architecture="Goguvik", vocab=size["vocab"], width=size["width"], streams=4,
                norm=dict(eps=1e-6), layers=out)


def qwen3_config(size: dict, layers: int) -> dict:
    return dict(QWEN3_4B, num_hidden_layers=layers, hidden_size=size["width"], intermediate_size=size["ff"],
                num_attention_heads=size["heads"], num_key_value_heads=size["kv_heads"], head_dim=128,
                vocab_size=size["vocab"])


def design_compare(args) -> int:
    """``--design goguvik``: prefill and decode throughput of Goguvik beside Qwen3 (the closest model
    this library has) at equal sizes, and each design's own kernels alone against their rooflines.
    Every number is timed on the device with CUDA events; the kernels alone run inside a CUDA graph,
    once per layer on that layer's own weights and cache.  Prints one JSON line."""
    import torch

    from starter_b200 import ops
    from starter_b200.config import config_from_dict
    from starter_b200.engine import ModelRunner, StepEntry, random_model

    pk = peaks()
    layers = args.layers if args.layers_given else 8
    batch, context, prompt_len = args.batch, 2048, PROMPT
    warmup, steps = max(args.warmup, 3), max(min(args.steps, 64), 1)
    sampler = ClockSampler()
    sampler.start()
    windows = []
    gen = torch.Generator().manual_seed(0)
    dev = torch.device("cuda:0")

    def timed(fn, reps):
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        t0 = time.monotonic()
        start.record()
        for _ in range(reps):
            fn()
        stop.record()
        torch.cuda.synchronize()
        windows.append((t0, time.monotonic()))
        return start.elapsed_time(stop) / reps

    def in_graph(calls):
        """Microseconds per call of ``calls`` (one per layer), captured together and replayed."""
        for c in calls:
            c()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for c in calls:
                c()
        graph.replay()
        return timed(graph.replay, 5) / len(calls) * 1e3

    def kernels_alone(model, runner, design, size):
        """Each design's own kernels, at the prompt's 2,048 rows and at the decode batch."""
        spec = model.spec
        blocks = [model.blocks[e.layer] for e in spec.schedule]
        writers = [(b, e.cache) for b, e in zip(blocks, spec.schedule) if e.writes_cache]
        cache = runner.cache
        w, heads, kvh = size["width"], size["heads"], size["kv_heads"]
        out = {}
        slots = [runner.open_sequence() for _ in range(batch)]
        for s in slots:
            runner.step([StepEntry(s, torch.randint(0, spec.vocab_size, (context,), generator=gen).tolist(), [])])
        for rows, name in ((prompt_len, "prompt"), (batch, "decode")):
            if rows == prompt_len:
                slot = runner.open_sequence()
                ctx = runner.make_context([StepEntry(slot, [1] * prompt_len, [])])
            else:
                ctx = runner.make_context([StepEntry(s, [1], []) for s in slots])
            x = (torch.randn(rows, w, device=dev) * 0.5).to(torch.bfloat16)
            kv_tokens = int(ctx.host["seq_kv_len"].sum())
            if design == "goguvik":
                streams = torch.randn(rows, spec.streams, w, device=dev)
                us = in_graph([lambda b=b: b.connection2.open(streams, ops_pending(b, x), b.norm2, torch.bfloat16) for b in blocks])
                moved = rows * w * (2 * spec.streams * 4 + 2 + 2)
                out[f"{name}: stream write + read + norm"] = dict(us=us, gbs=moved / us / 1e3)
                m = blocks[0].mixer
                proj = (torch.randn(rows, m.weight.shape[0], device=dev) * 0.5).to(torch.bfloat16)
                q = (torch.randn(rows, m.q_size, device=dev) * 0.5).to(torch.bfloat16)
                gate = proj[:, m.q_size:m.q_size + m.gate_size]
                sp = m.spec

                def prepare(b, e):
                    k, v = cache.entry_pages(e)
                    return ops.diff_prepare(proj, b.mixer.bias, heads, kvh, sp.head_dim, sp.value_dim, m.gate_size,
                                            (0.5, 128), ctx.tok_pos, ctx.tok_slot, cache.block_table, k, v)

                def attend(b, e):
                    k, v = cache.entry_pages(e)
                    return ops.diff_attention_step(q, gate, k, v, cache.block_table, ctx, heads, kvh, sp.head_dim,
                                                   sp.value_dim, sp.scale, 0.4, 0.7, 1e-6)

                us = in_graph([lambda b=b, e=e: prepare(b, e) for b, e in writers])
                moved = rows * 2 * (2 * m.q_size + 2 * (m.k_size + m.v_size))
                out[f"{name}: bias, temperature, cache write"] = dict(us=us, gbs=moved / us / 1e3)
                us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in writers])
                flops = heads * (4 * sp.head_dim + 4 * sp.value_dim)
            else:
                res = x.clone()
                us = in_graph([lambda b=b: ops.rmsnorm(res, b.norm1.weight, b.norm1.spec.eps, delta=x) for b in blocks])
                out[f"{name}: residual sum + norm"] = dict(us=us, gbs=rows * w * 2 * 4 / us / 1e3)
                m = blocks[0].mixer
                sp = m.spec
                qkv = (torch.randn(rows, m.qkv.shape[0], device=dev) * 0.5).to(torch.bfloat16)
                rot = m.position.rotation()

                def attend(b, e):
                    k, v = cache.entry_pages(e)
                    if rows == batch:
                        return ops.attention_decode_qkv(qkv, k, v, cache.block_table, ctx.seq_slot, ctx.seq_kv_len, heads,
                                                        kvh, sp.head_dim, sp.scale, None, b.mixer.q_norm, b.mixer.k_norm,
                                                        sp.qk_norm_eps, rot.cos, rot.sin, write_cache=True,
                                                        kv_hint=ctx.max_kv_len)
                    qq = ops.qk_norm_rope_store(qkv, heads, kvh, sp.head_dim, b.mixer.q_norm, b.mixer.k_norm,
                                                sp.qk_norm_eps, rot.cos, rot.sin, ctx.tok_pos, ctx.tok_slot,
                                                cache.block_table, k, v)
                    return ops.attention_prefill(qq, k, v, cache.block_table, ctx.seq_slot, ctx.seq_q_start,
                                                 ctx.seq_q_len, ctx.seq_kv_len, ctx.tile_seq, ctx.tile_first, heads, kvh,
                                                 sp.head_dim, sp.scale, None, max_q_len=ctx.max_q_len,
                                                 blocks=(ctx.block_seq, ctx.block_first))

                if rows == prompt_len:
                    def store(b, e):
                        k, v = cache.entry_pages(e)
                        return ops.qk_norm_rope_store(qkv, heads, kvh, sp.head_dim, b.mixer.q_norm, b.mixer.k_norm,
                                                      sp.qk_norm_eps, rot.cos, rot.sin, ctx.tok_pos, ctx.tok_slot,
                                                      cache.block_table, k, v)
                    us_store = in_graph([lambda b=b, e=e: store(b, e) for b, e in writers])
                    moved = rows * 2 * (qkv.shape[1] + heads * sp.head_dim + 2 * kvh * sp.head_dim)
                    out[f"{name}: head norm, rotation, cache write"] = dict(us=us_store, gbs=moved / us_store / 1e3)
                us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in writers])
                if rows == prompt_len:
                    us -= us_store
                flops = heads * 4 * sp.head_dim
            if rows == prompt_len:
                pairs = prompt_len * (prompt_len + 1) / 2
                tf = flops * pairs / us / 1e6
                out[f"{name}: attention"] = dict(us=us, tflops=tf, frac_of_bf16_peak=tf / pk["bf16_tflops"])
                runner.close_sequence(slot)
            else:
                kv_bytes = cache.bytes_per_token() // len({e.cache for e in spec.schedule if e.writes_cache}) * kv_tokens
                out[f"{name}: attention"] = dict(us=us, gbs=kv_bytes / us / 1e3, frac_of_copy_peak=kv_bytes / us / 1e3 / pk["hbm_gbs"])
            for slot_, length in zip(ctx.host["seq_slot"].tolist(), ctx.host["seq_kv_len"].tolist()):
                if rows == batch:
                    cache.lengths[slot_] = length - 1       # the context made above counted a token that no step ran
        for s in slots:
            runner.close_sequence(s)
        return {k: {a: round(b, 4 if "frac" in a else 1) for a, b in v.items()} for k, v in out.items()}

    def ops_pending(block, y):
        from starter_b200.parts import Pending
        return Pending(y, block.connection1, block.mixer.deferred_bias)

    results = {}
    for size_name in (args.design_sizes.split(",") if args.design_sizes else list(DESIGN_SIZES)):
        size = DESIGN_SIZES[size_name]
        row = {"layers": layers}
        for design, raw in (("goguvik", goguvik_config(size, layers)), ("qwen3", qwen3_config(size, layers))):
            config = config_from_dict(raw)
            model = random_model(config, seed=0, dtype="bfloat16")
            vocab = model.spec.vocab_size
            runner = ModelRunner(model, max_tokens=(batch + 1) * (context + 256) + prompt_len, max_sequences=batch + 2)
            prompt = torch.randint(0, vocab, (prompt_len,), generator=gen).tolist()

            def prefill_once():
                slot = runner.open_sequence()
                runner.step([StepEntry(slot, prompt, [prompt_len - 1])])
                runner.close_sequence(slot)

            for _ in range(warmup):
                prefill_once()
            prefill_ms = timed(prefill_once, 5)
            slots = [runner.open_sequence() for _ in range(batch)]
            for s in slots:
                runner.reserve(s, context + 256)
                runner.step([StepEntry(s, torch.randint(0, vocab, (context,), generator=gen).tolist(), [])])
            entries = [StepEntry(s, [1], [0]) for s in slots]

            def one():
                runner.decode_tokens(entries, [0.0] * batch, [0] * batch)

            for _ in range(warmup):
                one()
            decode_ms = timed(one, steps)
            for s in slots:
                runner.close_sequence(s)
            runner.check_status()
            step_bytes = model.step_weight_bytes() + runner.cache.bytes_per_token() * batch * context
            row[design] = {
                "prefill_tok_s": round(prompt_len / prefill_ms * 1e3, 1), "prefill_ms": round(prefill_ms, 3),
                "decode_tok_s": round(batch / decode_ms * 1e3, 1), "decode_ms_per_step": round(decode_ms, 4),
                "decode_frac_of_copy_peak": round(step_bytes / (decode_ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4),
                "weight_mb_per_step": round(model.step_weight_bytes() / 1e6, 1),
                "kernels": kernels_alone(model, runner, design, size),
            }
            del runner, model
            torch.cuda.empty_cache()
        results[size_name] = row
    print(json.dumps({
        "metric": "prefill tok/s at 2,048 tokens and decode tok/s at batch %d, context 2,048: Goguvik beside Qwen3 at "
                  "equal sizes (BF16, random weights)" % batch,
        "unit": "tok/s", "n_gpus": 1, "dtype": "bf16", "steps": steps, "warmup": warmup,
        "data": "synthetic: random weights, uniform random token ids", "peaks": pk,
        "sizes": {k: DESIGN_SIZES[k] for k in results}, "results": results, "clocks": sampler.stop(windows)}))
    return 0


def qwen3_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                        in_graph, bw, tc):
    """Qwen3's own kernels alone at ``rows`` rows (the prompt's, or the decode batch), once per layer inside a
    CUDA graph: what the design comparisons set their kernels beside."""
    w = size["width"]
    heads, kvh = size["heads"], size["kv_heads"]
    res = x.clone()
    us = in_graph([lambda b=b: ops.rmsnorm(res, b.norm1.weight, b.norm1.spec.eps, delta=x) for b in blocks])
    out[f"{name}: residual sum + norm"] = bw(us, rows * w * 2 * 4)
    m = blocks[0].mixer
    sp = m.spec
    qkv = rnd(rows, m.qkv.shape[0])
    rot = m.position.rotation()
    entries = [(b, e.cache) for b, e in zip(blocks, spec.schedule)]

    def store(b, e):
        k, v = cache.entry_pages(e)
        return ops.qk_norm_rope_store(qkv, heads, kvh, sp.head_dim, b.mixer.q_norm, b.mixer.k_norm, sp.qk_norm_eps,
                                      rot.cos, rot.sin, ctx.tok_pos, ctx.tok_slot, cache.block_table, k, v)

    def attend(b, e):
        k, v = cache.entry_pages(e)
        if rows == batch:
            return ops.attention_decode_qkv(qkv, k, v, cache.block_table, ctx.seq_slot, ctx.seq_kv_len, heads, kvh,
                                            sp.head_dim, sp.scale, None, b.mixer.q_norm, b.mixer.k_norm,
                                            sp.qk_norm_eps, rot.cos, rot.sin, write_cache=True, kv_hint=ctx.max_kv_len)
        return ops.attention_prefill(store(b, e), k, v, cache.block_table, ctx.seq_slot, ctx.seq_q_start,
                                     ctx.seq_q_len, ctx.seq_kv_len, ctx.tile_seq, ctx.tile_first, heads, kvh,
                                     sp.head_dim, sp.scale, None, max_q_len=ctx.max_q_len,
                                     blocks=(ctx.block_seq, ctx.block_first))

    us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in entries])
    if rows == prompt_len:
        us_store = in_graph([lambda b=b, e=e: store(b, e) for b, e in entries])
        out[f"{name}: head norm, rotation, cache write"] = bw(us_store, rows * 2 * (qkv.shape[1] + (heads + 2 * kvh) * sp.head_dim))
        out[f"{name}: attention"] = tc(us - us_store, heads * 4 * sp.head_dim * prompt_len * (prompt_len + 1) / 2)
    else:
        out[f"{name}: attention"] = bw(us, batch * (context + 1) * 2 * kvh * sp.head_dim * 2)
    ff = blocks[0].feed_forward
    us = in_graph([lambda b=b: b.feed_forward(x, None) for b in blocks])
    flops = rows * 3 * ff.spec.intermediate_size * w * 2
    if rows == prompt_len:
        out[f"{name}: feed-forward (gate, up, down)"] = tc(us, flops)
    else:
        out[f"{name}: feed-forward (gate, up, down)"] = bw(us, 3 * ff.spec.intermediate_size * w * 2)


def kesedra_config(size: dict, layers: int) -> dict:
    """Kesedra at ``size``: of every four layers a recurrent one with a dense feed-forward, latent attention
    with routed experts, a recurrent one with routed experts, and latent attention over the second layer's
    latent with a dense feed-forward.  Recurrent heads of 64 channels; latent attention with 128 plain + 64
    rotated query/key entries and values of 128 a head over a latent of 512, a window of 1,024; 16 experts of a
    quarter of the dense width, four a token (as many active feed-forward rows as the dense layer)."""
    w, out = size["width"], []
    moe = dict(kind="moe", expert=dict(ff=size["ff"] // 4 // 64 * 64, limit=7.0), router=dict(experts=16, top=4))
    dense = dict(kind="dense", ff=size["ff"])
    for i in range(layers):
        if i % 2 == 0:
            mixer, kind = dict(heads=w // 64, dim=64, decay_rank=64), "wkv"
        else:
            mixer, kind = dict(heads=size["heads"], dim=128, rot_dim=64, vdim=128, q_rank=w * 3 // 4 // 64 * 64, kv_rank=512,
                               scale=192 ** -0.5, mask=dict(size=1024), rot=dict(base=10000.0, dims=64)), "latent_attention"
            if i % 4 == 3:
                mixer["kv_from"] = i - 2
        out.append(dict(type=kind, mixer=mixer, mlp=dense if i % 4 in (0, 3) else moe))
    return dict(architecture="Kesedra", vocab=size["vocab"], width=w, embedding=dict(scale=16.0), norm=dict(eps=1e-5),
                layers=out)


def kesedra_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                          in_graph, bw, tc):
    """Kesedra's own kernels alone at ``rows`` rows, once per layer inside a CUDA graph."""
    import torch

    w, dev, bf = size["width"], x.device, x.dtype
    res = torch.randn(rows, w, device=dev)
    us = in_graph([lambda b=b: ops.residual_norm(res, bf, 1e-5, (x, b.norm1b.weight, None, 1e-5), b.norm2.weight)
                   for b in blocks])
    out[f"{name}: post-norm + residual sum + norm"] = bw(us, rows * w * (2 + 4 + 4 + 2))
    rec = [(b, e.cache) for b, e in zip(blocks, spec.schedule) if b.mixer.spec.kind == "wkv"]
    m = rec[0][0].mixer
    hd, heads, dim = m.inner, m.spec.num_heads, m.spec.head_dim
    r, k, v, g = (rnd(rows, hd) for _ in range(4))
    xd = torch.rand(rows, hd, device=dev)
    us = in_graph([lambda b=b, e=e: ops.token_shift(x, cache.entry_state(e), b.mixer.mu, ctx.tok_slot) for b, e in rec])
    out[f"{name}: token shift (five mixes)"] = bw(us, rows * w * 2 * 6)
    us = in_graph([lambda b=b, e=e: ops.wkv_scan(r, k, v, xd, b.mixer.u, g, b.mixer.gain, cache.entry_state(e),
                                                  x, ctx.seq_slot, ctx.seq_q_start, ctx.seq_q_len, heads, dim, 1e-5)
                   for b, e in rec])
    state_bytes = ctx.n_seqs * heads * dim * dim * 4 * 2
    d = bw(us, rows * hd * (5 * 2 + 4) + state_bytes)
    d["gflops"] = rows * heads * dim * dim * 6 / us / 1e3
    out[f"{name}: recurrence (state walk, head norm, gate)"] = d
    att = [(b, e.cache, e.writes_cache) for b, e in zip(blocks, spec.schedule) if b.mixer.spec.kind == "latent_attention"]
    m = att[0][0].mixer
    sp = m.spec
    proj = rnd(rows, m.down.shape[0])
    cos, sin = ops.latent_tables(m.position.rotation(), sp.position.dims)
    own = [(b, e) for b, e, wr in att if wr]
    us = in_graph([lambda b=b, e=e: ops.latent_prepare(proj, b.mixer.q_gain, b.mixer.kv_gain, 1e-5, cos, sin, ctx.tok_pos,
                                                        ctx.tok_slot, cache.block_table, cache.entry_pages(e)[0], sp.q_rank,
                                                        sp.kv_rank, sp.rot_dim, sp.position.dims) for b, e in own])
    out[f"{name}: latent norms, rotation, cache write"] = bw(us, rows * 2 * (proj.shape[1] + sp.q_rank + m.row))
    qa = rnd(rows, sp.num_heads, m.row)
    us = in_graph([lambda b=b, e=e: ops.latent_attention_step(qa, cache.entry_pages(e)[0], cache.block_table, ctx,
                                                               sp.num_heads, sp.kv_rank, sp.rot_dim, sp.scale, sp.window)
                   for b, e in own])
    if rows == prompt_len:
        seen = sum(min(p + 1, sp.window) for p in range(prompt_len))
        out[f"{name}: attention"] = tc(us, sp.num_heads * 2 * (m.row + sp.kv_rank) * seen)
    else:
        out[f"{name}: attention"] = bw(us, batch * min(context + 1, sp.window) * m.row * 2)
    routed = [b for b in blocks if getattr(b.feed_forward, "last_ids", "no") != "no"]
    ff = routed[0].feed_forward
    fs = ff.spec
    ids, weights = ops.moe_route(x, ff.router, ff.router_bias, fs.top)
    us = in_graph([lambda b=b: ops.moe_route(x, b.feed_forward.router, b.feed_forward.router_bias, fs.top) for b in routed])
    out[f"{name}: router"] = bw(us, rows * w * 2 + fs.experts * w * 4)
    us = in_graph([lambda b=b: ops.moe_experts(x, ids, weights, b.feed_forward.gate_up, b.feed_forward.down, fs.limit)
                   for b in routed])
    flops = rows * fs.top * 3 * fs.intermediate_size * w * 2
    if rows == prompt_len:
        out[f"{name}: experts (gate, up, down, sum)"] = tc(us, flops)
    else:
        used = min(fs.experts, rows * fs.top)
        out[f"{name}: experts (gate, up, down, sum)"] = bw(us, used * 3 * fs.intermediate_size * w * 2)


def korurax_config(size: dict, layers: int) -> dict:
    """Korurax at ``size``: latent attention with a dense clamped feed-forward and attention with a sink with
    routed squared-relu experts, in turn.  Latent attention with 128 plain + 64 rotated query/key entries and
    values of 128 a head over a latent of 512; the other attention with keys and values of 128 and chunks of
    3,072 positions (longer than the timed contexts, so that it sees as many keys as Qwen3's); 16 experts of
    three eighths of the dense width, four a token (as many active feed-forward rows as the gated dense layer)."""
    w, out = size["width"], []
    moe = dict(kind="moe", expert=dict(ff=size["ff"] * 3 // 8 // 64 * 64), router=dict(experts=16, top=4, scale=2.5))
    dense = dict(kind="dense", ff=size["ff"], limit=7.0)
    for i in range(layers):
        if i % 2 == 0:
            mixer, kind = dict(heads=size["heads"], dim=128, rot_dim=64, vdim=128, q_rank=w * 3 // 4 // 64 * 64, kv_rank=512,
                               scale=192 ** -0.5, rot=dict(base=10000.0, dims=64)), "latent_attention"
        else:
            mixer, kind = dict(heads=size["heads"], kv_heads=size["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5,
                               mask=dict(size=3072)), "attention"
        out.append(dict(type=kind, mixer=mixer, mlp=dense if i % 2 == 0 else moe))
    return dict(architecture="Korurax", vocab=size["vocab"], width=w, norm=dict(eps=1e-5), residual_mult=0.5,
                logit_softcap=30.0, layers=out)


def korurax_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                          in_graph, bw, tc):
    """Korurax's own kernels alone at ``rows`` rows, once per layer inside a CUDA graph."""
    import torch

    w, dev, bf = size["width"], x.device, x.dtype
    levels = max(b.levels for b in blocks)
    history = torch.randn(levels, rows, w, device=dev)
    base, dst = torch.randn(rows, w, device=dev), torch.empty(rows, w, device=dev)
    us = in_graph([lambda b=b: ops.depth_step(base, bf, x, 0.5, dst=dst, norm=b.norm2.for_kernel()) for b in blocks])
    out[f"{name}: sum inside a layer + norm"] = bw(us, rows * w * (4 + 2 + 4 + 2))
    us = in_graph([lambda b=b: ops.depth_step(base, bf, x, 0.5, history, b.connection.weights, dst, b.norm1.for_kernel())
                   for b in blocks])
    mean_levels = sum(b.levels for b in blocks) / len(blocks)
    out[f"{name}: layer end (sum, filing, sum over depth) + norm"] = bw(us, rows * w * (4 + 2 + 4 + 4 * (mean_levels - 1) + 4 + 2))
    att = [(b, e.cache) for b, e in zip(blocks, spec.schedule) if b.mixer.spec.kind == "sink_attention"]
    m = att[0][0].mixer
    sp = m.spec
    proj = rnd(rows, m.qkvg.shape[0])

    def prepare(b, e):
        k, v = cache.entry_pages(e)
        return ops.sink_prepare(proj, sp.num_heads, sp.num_kv_heads, sp.head_dim, sp.value_dim, ctx.tok_pos, ctx.tok_slot,
                                cache.block_table, k, v)

    gate = prepare(*att[0])
    us = in_graph([lambda b=b, e=e: prepare(b, e) for b, e in att])
    kv_row = sp.num_kv_heads * (sp.head_dim + sp.value_dim)
    out[f"{name}: cache write + gates"] = bw(us, rows * (2 * 2 * kv_row + 2 * sp.num_heads + 4 * sp.num_heads))

    def attend(b, e):
        k, v = cache.entry_pages(e)
        return ops.sink_attention_step(proj, k, v, cache.block_table, ctx, sp.num_heads, sp.num_kv_heads, sp.head_dim,
                                       sp.value_dim, sp.scale, b.mixer.penalty, b.mixer.sink, gate, sp.chunk, sp.window)

    us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in att])
    if rows == prompt_len:
        seen = sum(p % sp.chunk + 1 for p in range(prompt_len))
        out[f"{name}: attention"] = tc(us, sp.num_heads * 2 * (sp.head_dim + sp.value_dim) * seen)
    else:
        out[f"{name}: attention"] = bw(us, batch * (context % sp.chunk + 1) * kv_row * 2)
    lat = [(b, e.cache) for b, e in zip(blocks, spec.schedule) if b.mixer.spec.kind == "latent_attention"]
    m = lat[0][0].mixer
    lp = m.spec
    down = rnd(rows, m.down.shape[0])
    rotation = m.position.rotation()
    cos, sin = ops.latent_tables(rotation, lp.position.dims)
    us = in_graph([lambda b=b, e=e: ops.latent_prepare(down, b.mixer.q_gain, b.mixer.kv_gain, 1e-5, cos, sin, ctx.tok_pos,
                                                        ctx.tok_slot, cache.block_table, cache.entry_pages(e)[0], lp.q_rank,
                                                        lp.kv_rank, lp.rot_dim, lp.position.dims, layout=rotation.layout)
                   for b, e in lat])
    out[f"{name}: latent norms, rotation, cache write"] = bw(us, rows * 2 * (down.shape[1] + lp.q_rank + m.row))
    qa = rnd(rows, lp.num_heads, m.row)
    us = in_graph([lambda b=b, e=e: ops.latent_attention_step(qa, cache.entry_pages(e)[0], cache.block_table, ctx, lp.num_heads,
                                                               lp.kv_rank, lp.rot_dim, lp.scale, None) for b, e in lat])
    if rows == prompt_len:
        out[f"{name}: latent attention"] = tc(us, lp.num_heads * 2 * (m.row + lp.kv_rank) * prompt_len * (prompt_len + 1) / 2)
    else:
        out[f"{name}: latent attention"] = bw(us, batch * (context + 1) * m.row * 2)
    dense = [b for b in blocks if b.feed_forward.spec.kind == "gated_clamped"]
    fd = dense[0].feed_forward.spec
    us = in_graph([lambda b=b: b.feed_forward(x, None) for b in dense])
    if rows == prompt_len:
        out[f"{name}: dense feed-forward (gate, up, down)"] = tc(us, rows * 3 * fd.intermediate_size * w * 2)
    else:
        out[f"{name}: dense feed-forward (gate, up, down)"] = bw(us, 3 * fd.intermediate_size * w * 2)
    routed = [b for b in blocks if b.feed_forward.spec.kind == "routed_experts"]
    ff = routed[0].feed_forward
    fs = ff.spec
    ids, weights = ops.moe_route(x, ff.router, None, fs.top, fs.scoring, fs.weight_scale)
    us = in_graph([lambda b=b: ops.moe_route(x, b.feed_forward.router, None, fs.top, fs.scoring, fs.weight_scale)
                   for b in routed])
    out[f"{name}: router"] = bw(us, rows * w * 2 + fs.experts * w * 4)
    us = in_graph([lambda b=b: ops.moe_experts(x, ids, weights, b.feed_forward.gate_up, b.feed_forward.down, 0.0, fs.expert)
                   for b in routed])
    if rows == prompt_len:
        out[f"{name}: experts (up, down, sum)"] = tc(us, rows * fs.top * 2 * fs.intermediate_size * w * 2)
    else:
        used = min(fs.experts, rows * fs.top)
        out[f"{name}: experts (up, down, sum)"] = bw(us, used * 2 * fs.intermediate_size * w * 2)


def bavedra_config(size: dict, layers: int) -> dict:
    """Bavedra at ``size``: of every four layers a delta-rule one with a dense feed-forward, a recurrent unit with
    routed experts, window attention beside a state-space recurrence with routed experts, and a delta-rule one with
    routed experts.  Delta heads of 128 x 128 (half as many query/key heads), a recurrent unit as wide as the model in
    blocks of 256, attention heads of 128 with a window of 1,024 and half of each head rotated, state-space heads of 64
    with a state of 128; 16 experts of a quarter of the dense width and four identity experts in four groups of which
    two are kept, four a token, a shared expert of the same size (about as many active feed-forward rows as the dense
    layer)."""
    w, out = size["width"], []
    inner = size["ff"] // 4 // 64 * 64
    moe = dict(kind="moe", expert=dict(ff=inner), shared=dict(ff=inner),
               router=dict(experts=16, top=4, identity=4, groups=dict(count=4, keep=2)))
    dense = dict(kind="dense", ff=size["ff"])
    delta = dict(heads=w // 128, kv_heads=max(1, w // 256), dim=128, vdim=128, conv=4)
    for i in range(layers):
        if i % 4 in (0, 3):
            mixer, kind = delta, "delta"
        elif i % 4 == 1:
            mixer, kind = dict(width=w, blocks=w // 256, conv=4), "rglru"
        else:
            mixer, kind = dict(left=dict(heads=size["heads"], kv_heads=size["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5,
                                         mask=dict(size=1024), rot=dict(base=1e6, dims=64)),
                               right=dict(heads=w // 64, vdim=64, state=128, groups=1, conv=4, norm_groups=1)), "parallel"
        out.append(dict(type=kind, mixer=mixer, mlp=dense if i % 4 == 0 else moe))
    return dict(architecture="Bavedra", vocab=size["vocab"], width=w, embedding=dict(scale=16.0), norm=dict(eps=1e-6),
                layers=out)


def bavedra_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                          in_graph, bw, tc):
    """Bavedra's own kernels alone at ``rows`` rows, once per layer inside a CUDA graph."""
    import torch

    w, dev, bf = size["width"], x.device, x.dtype
    res = torch.randn(rows, w, device=dev)
    us = in_graph([lambda b=b: ops.residual_norm(res, bf, 1e-6, (x, None, None, 0.0), b.norm1.weight) for b in blocks])
    out[f"{name}: residual sum + norm"] = bw(us, rows * w * (2 + 4 + 4 + 2))
    seqs = (ctx.seq_slot, ctx.seq_q_start, ctx.seq_q_len)
    n_seqs = ctx.n_seqs
    pairs = [(b, e.cache) for b, e in zip(blocks, spec.schedule)]

    # the delta rule
    rec = [(b, e) for b, e in pairs if b.mixer.spec.kind == "gated_delta"]
    m = rec[0][0].mixer
    sp = m.spec
    proj = rnd(rows, m.stacked.shape[0])
    conv_state = n_seqs * (sp.conv - 1) * m.convolved * 4 * 2
    us = in_graph([lambda b=b, e=e: ops.short_conv(proj, 0, m.convolved, b.mixer.conv, None, None, cache.entry_state(e), 0, *seqs,
                                                    ctx.max_q_len, "silu") for b, e in rec])
    out[f"{name}: short convolution + silu ({m.convolved} channels)"] = bw(us, rows * m.convolved * 4 + conv_state)
    qkv = rnd(rows, m.convolved)
    us = in_graph([lambda b=b, e=e: ops.state_scan("gated_delta", (qkv, 0), (qkv, m.qk), (qkv, 2 * m.qk),
                                                    (proj, m.convolved + m.inner + sp.num_heads), (proj, m.convolved + m.inner),
                                                    b.mixer.A_log, b.mixer.dt_bias, None, cache.entry_state(e),
                                                    (sp.conv - 1) * m.convolved, *seqs, sp.num_heads, sp.num_kv_heads,
                                                    sp.head_dim, sp.value_dim) for b, e in rec])
    state_bytes = n_seqs * sp.num_heads * sp.head_dim * sp.value_dim * 4 * 2
    d = bw(us, rows * (m.convolved * 2 + m.inner * 4) + state_bytes)
    d["gflops"] = rows * sp.num_heads * sp.head_dim * sp.value_dim * 8 / us / 1e3
    out[f"{name}: delta-rule recurrence (unit norms, state walk)"] = d
    o32 = torch.randn(rows, m.inner, device=dev)
    us = in_graph([lambda b=b: ops.group_norm_gate(o32, proj, m.convolved, b.mixer.gain, sp.num_heads, 1e-6, False, bf) for b, _ in rec])
    out[f"{name}: head norm + gate"] = bw(us, rows * m.inner * (4 + 2 + 2))

    # the recurrent unit
    rec = [(b, e) for b, e in pairs if b.mixer.spec.kind == "gated_linear_recurrence"]
    m = rec[0][0].mixer
    sp = m.spec
    c = sp.width
    proj = rnd(rows, 2 * c)
    u = rnd(rows, c)
    us = in_graph([lambda b=b, e=e: ops.short_conv(proj, c, c, b.mixer.conv, b.mixer.conv_bias, b.mixer.x_bias, cache.entry_state(e), 0,
                                                    *seqs, ctx.max_q_len) for b, e in rec])
    out[f"{name}: short convolution ({c} channels)"] = bw(us, rows * c * 4 + n_seqs * (sp.conv - 1) * c * 8)
    parts = u.view(rows, sp.blocks, m.block).transpose(0, 1)
    us = in_graph([lambda b=b: torch.bmm(parts, b.mixer.gates, out_dtype=torch.float32) for b, _ in rec])
    flops = rows * sp.blocks * m.block * 2 * m.block * 2
    out[f"{name}: gate logits (library batched product)"] = tc(us, flops) if rows == prompt_len else bw(us, 2 * c * m.block * 2)
    logits = torch.randn(sp.blocks, rows, 2 * m.block, device=dev)
    us = in_graph([lambda b=b, e=e: ops.glru_scan(u, logits, b.mixer.ra_bias, b.mixer.ri_bias, b.mixer.lam, sp.decay_scale, proj, 0,
                                                   b.mixer.y_bias, cache.entry_state(e), (sp.conv - 1) * c, *seqs, ctx.max_q_len)
                   for b, e in rec])
    out[f"{name}: gated linear recurrence (gates, decay, walk, gelu branch)"] = bw(us, rows * c * (2 + 8 + 2 + 2) + n_seqs * c * 8)

    # window attention beside the state-space recurrence
    par = [(b, e) for b, e in pairs if b.mixer.spec.kind == "parallel"]
    m = par[0][0].mixer.sides["right"]
    sp = m.spec
    proj = rnd(rows, m.w_in.shape[0])
    us = in_graph([lambda b=b, e=e: ops.short_conv(proj, m.inner, m.convolved, b.mixer.sides["right"].conv,
                                                    b.mixer.sides["right"].conv_bias, None, cache.entry_state(e), 0, *seqs,
                                                    ctx.max_q_len, "silu") for b, e in par])
    out[f"{name}: short convolution + silu ({m.convolved} channels)"] = bw(us, rows * m.convolved * 4 + n_seqs * (sp.conv - 1) * m.convolved * 8)
    xbc = rnd(rows, m.convolved)
    us = in_graph([lambda b=b, e=e: ops.state_scan("state_space", (xbc, m.inner + m.bc), (xbc, m.inner), (xbc, 0),
                                                    (proj, m.inner + m.convolved), None, b.mixer.sides["right"].A_log,
                                                    b.mixer.sides["right"].dt_bias, b.mixer.sides["right"].D, cache.entry_state(e),
                                                    (sp.conv - 1) * m.convolved, *seqs, sp.num_heads, sp.groups, sp.state,
                                                    sp.head_dim) for b, e in par])
    state_bytes = n_seqs * sp.num_heads * sp.state * sp.head_dim * 4 * 2
    d = bw(us, rows * (m.convolved * 2 + m.inner * 4) + state_bytes)
    d["gflops"] = rows * sp.num_heads * sp.state * sp.head_dim * 5 / us / 1e3
    out[f"{name}: state-space recurrence (state walk)"] = d
    o32 = torch.randn(rows, m.inner, device=dev)
    us = in_graph([lambda b=b: ops.group_norm_gate(o32, proj, 0, b.mixer.sides["right"].gain, sp.norm_groups, 1e-6, True, bf)
                   for b, _ in par])
    out[f"{name}: gate + norm in groups"] = bw(us, rows * m.inner * (4 + 2 + 2))
    a = par[0][0].mixer.sides["left"]
    sp = a.spec
    heads, kvh, dim = sp.num_heads, sp.num_kv_heads, sp.head_dim
    proj = rnd(rows, a.qkvg.shape[0])
    cos, sin, dims = ops.sink_tables(a.position.rotation(), dim)

    def prepare(b, e):
        k, v = cache.entry_pages(e)
        ops.sink_prepare_rot(proj, heads, kvh, dim, dim, ctx.tok_pos, ctx.tok_slot, cache.block_table, k, v, cos, sin, dims,
                             values_from_keys=True)

    def attend(b, e):
        k, v = cache.entry_pages(e)
        return ops.sink_attention_step(proj, k, v, cache.block_table, ctx, heads, kvh, dim, dim, sp.scale, None,
                                       b.mixer.sides["left"].sink, None, None, sp.window)

    us = in_graph([lambda b=b, e=e: prepare(b, e) for b, e in par])
    out[f"{name}: rotation of queries and keys, cache write"] = bw(us, rows * 2 * (2 * heads * dim + 3 * kvh * dim))
    us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in par])
    if rows == prompt_len:
        seen = sum(min(p + 1, sp.window) for p in range(prompt_len))
        out[f"{name}: attention"] = tc(us, heads * 4 * dim * seen)
    else:
        out[f"{name}: attention"] = bw(us, batch * min(context + 1, sp.window) * 2 * kvh * dim * 2)
    us = in_graph([lambda b=b: ops.norm_pair_mean(x, x, b.mixer.gains["left"], b.mixer.gains["right"], 1e-6) for b, _ in par])
    out[f"{name}: two norms and their mean"] = bw(us, rows * w * 2 * 3)

    # routed experts
    routed = [b for b in blocks if getattr(b.feed_forward, "last_ids", "no") != "no"]
    ff = routed[0].feed_forward
    fs = ff.spec
    ids, weights, gate = ops.moe_route_all(x, ff.router, ff.correction, fs.top, fs.group_count, fs.group_keep, shared_gate=True)
    us = in_graph([lambda b=b: ops.moe_route_all(x, b.feed_forward.router, b.feed_forward.correction, fs.top, fs.group_count,
                                                 fs.group_keep, shared_gate=True) for b in routed])
    out[f"{name}: router"] = bw(us, rows * w * 2 + ff.router.shape[0] * w * 4)
    shared = rnd(rows, w)
    us = in_graph([lambda b=b: ops.moe_experts(x, ids, weights, b.feed_forward.gate_up, b.feed_forward.down, 0.0, "gated_silu",
                                               identity=True, shared=shared, shared_gate=gate) for b in routed])
    real = float((ids < fs.experts).float().mean())
    flops = rows * fs.top * real * 3 * fs.intermediate_size * w * 2
    if rows == prompt_len:
        out[f"{name}: experts (gate, up, down, sum with identity and shared rows)"] = tc(us, flops)
    else:
        used = min(fs.experts, int(rows * fs.top * real) or 1)
        out[f"{name}: experts (gate, up, down, sum with identity and shared rows)"] = bw(us, used * 3 * fs.intermediate_size * w * 2)
    dense = [b for b in blocks if getattr(b.feed_forward.spec, "kind", "") == "dense_biased"]
    us = in_graph([lambda b=b: b.feed_forward(x, None) for b in dense])
    fd = dense[0].feed_forward.spec
    if rows == prompt_len:
        out[f"{name}: dense feed-forward (up, squared relu, down)"] = tc(us, rows * 2 * fd.intermediate_size * w * 2)
    else:
        out[f"{name}: dense feed-forward (up, squared relu, down)"] = bw(us, 2 * fd.intermediate_size * w * 2)


def bavedra_compare(args) -> int:
    """Beside Kesedra: the closest design this library has (a recurrence with a matrix state per head, attention
    with a window, routed experts, a 32-bit residual stream)."""
    return compare_with_qwen3(args, "bavedra", "Bavedra", bavedra_config, bavedra_kernels_alone, ["2048"],
                              beside=("kesedra", "Kesedra", kesedra_config, kesedra_kernels_alone))


def setotar_config(size: dict, layers: int) -> dict:
    """Setotar at ``size``: of every four layers an attention over all keys (its queries and keys normed over their
    rows, 64 of 128 entries rotated, stretched by parts), two window attentions of 1,024 keys that keep the first four,
    with biases, three taps, unit values and capped scores, each beside a forget-write recurrence with states of 128 x
    128, and an attention that reads the first one's keys and values; four streams; 16 experts of a quarter of the
    dense width, four a token, in every layer."""
    w, out = size["width"], []
    moe = dict(kind="moe", expert=dict(ff=size["ff"] // 4 // 64 * 64), router=dict(experts=16, top=4))
    heads = dict(heads=size["heads"], kv_heads=size["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5)
    full = dict(heads, rot=dict(base=1e6, dims=64, scaling=dict(factor=4.0, original=8192, fast=32.0, slow=1.0)))
    side = dict(left=dict(heads, conv=3, mask=dict(size=1024, keep_first=4), softcap=50.0,
                          rot=dict(base=1e4, dims=64, scaling=dict(factor=2.0))),
                right=dict(heads=w // 128, dim=128, vdim=128), left_scale=0.7, right_scale=0.7)
    for i in range(layers):
        if i % 4 in (1, 2):
            out.append(dict(type="parallel", mixer=side, mlp=moe))
        else:
            out.append(dict(type="attention", mixer=full if i % 4 == 0 else dict(full, kv_from=i - 3), mlp=moe))
    return dict(architecture="Setotar", vocab=size["vocab"], width=w, streams=4, norm=dict(eps=1e-6), layers=out)


def setotar_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                          in_graph, bw, tc):
    """Setotar's own kernels alone at ``rows`` rows, once per layer inside a CUDA graph."""
    import torch

    w, dev, bf, n_streams = size["width"], x.device, x.dtype, spec.streams
    streams = torch.randn(rows, n_streams, w, device=dev) * 0.1
    us = in_graph([lambda b=b: ops.hyper_step(streams, bf, (x, b.connection1.mix * 0.1, b.connection1.out, None, b.connection1.scale),
                                              b.connection1.read, b.norm1.parameters()) for b in blocks])
    out[f"{name}: stream write, read + norm ({n_streams} streams)"] = bw(us, rows * w * (2 + 8 * n_streams + 2))
    seqs = (ctx.seq_slot, ctx.seq_q_start, ctx.seq_q_len)
    n_seqs = ctx.n_seqs
    pairs = [(b, e) for b, e in zip(blocks, spec.schedule)]

    def attention(title, chosen, a_of):
        a = a_of(chosen[0][0])
        sp = a.spec
        heads, kvh, dim, vdim = sp.num_heads, sp.num_kv_heads, sp.head_dim, sp.value_dim
        proj = rnd(rows, a.qkvg.shape[0])
        if a.taps is not None:
            us = in_graph([lambda b=b, e=e: ops.short_conv(proj, 0, a.convolved, a_of(b).taps, None, a_of(b).biases, cache.entry_state(e.cache),
                                                            a_of(b).state_at, *seqs, ctx.max_q_len) for b, e in chosen])
            state = n_seqs * (sp.conv - 1) * a.convolved * 8
            out[f"{name}: bias + short convolution ({a.convolved} channels)"] = bw(us, rows * a.convolved * 4 + state)

        def prepare(b, e):
            k, v = cache.entry_pages(e.cache)
            ops.sink_prepare_norm(proj, heads, kvh, dim, vdim, ctx.tok_pos, ctx.tok_slot, cache.block_table, k, v,
                                  a.position.rotation(), a_of(b).row_norm, sp.unit_values, sp.norm_eps)

        def attend(b, e):
            k, v = cache.entry_pages(e.cache)
            return ops.sink_attention_step(proj, k, v, cache.block_table, ctx, heads, kvh, dim, vdim, sp.scale, None, None, None, None,
                                           sp.window, sp.keep_first, sp.softcap)

        us = in_graph([lambda b=b, e=e: prepare(b, e) for b, e in chosen])
        turned = 2 * heads * dim if sp.row_norm else heads * sp.position.dims * 2
        out[f"{name}: {title}: norms, rotation, cache write"] = bw(us, rows * 2 * (turned + 2 * kvh * (dim + vdim)))
        us = in_graph([lambda b=b, e=e: attend(b, e) for b, e in chosen])
        span = lambda p: p + 1 if sp.window is None else min(p + 1, sp.window + sp.keep_first)  # noqa: E731
        if rows == prompt_len:
            out[f"{name}: {title}: attention"] = tc(us, heads * 2 * (dim + vdim) * sum(span(p) for p in range(prompt_len)))
        else:
            out[f"{name}: {title}: attention"] = bw(us, batch * span(context) * kvh * (dim + vdim) * 2)

    attention("all keys", [(b, e) for b, e in pairs if b.mixer.spec.kind == "sink_attention" and e.writes_cache], lambda b: b.mixer)
    par = [(b, e) for b, e in pairs if b.mixer.spec.kind == "parallel"]
    attention("window, kept keys, cap", par, lambda b: b.mixer.sides["left"])
    m = par[0][0].mixer.sides["right"]
    sp = m.spec
    proj = rnd(rows, m.stacked.shape[0])
    us = in_graph([lambda b=b, e=e: ops.state_scan("forget_write", (proj, 0), (proj, m.qk), (proj, 2 * m.qk), None, None,
                                                    b.mixer.sides["right"].lower, b.mixer.sides["right"].f_bias, None,
                                                    cache.entry_state(e.cache), b.mixer.sides["right"].state_at, *seqs, sp.num_heads,
                                                    sp.num_heads, sp.head_dim, sp.value_dim) for b, e in par])
    d = bw(us, rows * (2 * m.qk * 2 + m.inner * 6) + n_seqs * sp.num_heads * sp.head_dim * sp.value_dim * 4 * 2)
    d["gflops"] = rows * sp.num_heads * sp.head_dim * sp.value_dim * 5 / us / 1e3
    out[f"{name}: forget-write recurrence (gate, state walk)"] = d
    o32 = torch.randn(rows, m.inner, device=dev)
    us = in_graph([lambda b=b: ops.group_norm_gate(o32, None, 0, b.mixer.sides["right"].gain, sp.num_heads, 1e-6, False, bf)
                   for b, _ in par])
    out[f"{name}: head norm"] = bw(us, rows * m.inner * (4 + 2))
    us = in_graph([lambda b=b: ops.scaled_sum(x, x, 0.7, 0.7) for b, _ in par])
    out[f"{name}: scaled sum of two mixers"] = bw(us, rows * w * 2 * 3)
    ff = blocks[0].feed_forward
    fs = ff.spec
    ids, weights = ops.moe_route(x, ff.router, None, fs.top, fs.scoring)
    us = in_graph([lambda b=b: ops.moe_route(x, b.feed_forward.router, None, fs.top, fs.scoring) for b in blocks])
    out[f"{name}: router"] = bw(us, rows * w * 2 + ff.router.shape[0] * w * 4)
    us = in_graph([lambda b=b: ops.moe_experts(x, ids, weights, b.feed_forward.gate_up, b.feed_forward.down, 0.0, "gated_silu",
                                               weigh_input=True) for b in blocks])
    if rows == prompt_len:
        out[f"{name}: experts (gate, up, down, sum)"] = tc(us, rows * fs.top * 3 * fs.intermediate_size * w * 2)
    else:
        used = int(torch.unique(ids).numel())
        out[f"{name}: experts (gate, up, down, sum)"] = bw(us, used * 3 * fs.intermediate_size * w * 2)


def setotar_compare(args) -> int:
    """Beside Bavedra: the closest design this library has (a window attention beside a recurrence with a matrix state
    per head, rotated keys, routed experts, a 32-bit residual)."""
    return compare_with_qwen3(args, "setotar", "Setotar", setotar_config, setotar_kernels_alone, ["2048"],
                              beside=("bavedra", "Bavedra", bavedra_config, bavedra_kernels_alone))


def salulorn_config(size: dict, layers: int) -> dict:
    """Salulorn at ``size``: a recurrence, window attention and latent attention in turn, each beside a dense gated
    feed-forward, the first two layers passed through twice (``layers`` runs of ``layers - 2`` stored layers).  Recurrent
    states of 128 x 128 with decays of rank 16; attention heads of 128 with biases, three taps, the whole head rotated, a
    window of 1,024 and a cap; latent attention with 128 plain + 64 rotated query/key entries and values of 128 a head
    over a latent of 512, stretched by parts."""
    w, out = size["width"], []
    dense = dict(kind="dense", ff=size["ff"])
    kinds = (("gla", dict(heads=w // 128, dim=128, vdim=128, tau=16.0, decay_rank=16)),
             ("attention", dict(heads=size["heads"], kv_heads=size["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5, conv=3,
                                mask=dict(size=1024), rot=dict(base=1e6, dims=128), softcap=50.0)),
             ("latent_attention", dict(heads=size["heads"], dim=128, rot_dim=64, vdim=128, q_rank=w * 3 // 4 // 64 * 64, kv_rank=512,
                                       scale=192 ** -0.5, rot=dict(base=1e4, dims=64, scaling=dict(
                                           factor=4.0, original=8192, fast=32.0, slow=1.0)))))
    for i in range(layers - 2):
        kind, mixer = kinds[i % 3]
        out.append(dict(type=kind, mixer=mixer, mlp=dense))
    return dict(architecture="Salulorn", vocab=size["vocab"], width=w, norm=dict(eps=1e-6), layers=out,
                loop=dict(start=0, stop=2, times=2))


def salulorn_kernels_alone(ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                           in_graph, bw, tc):
    """Salulorn's own kernels alone at ``rows`` rows, once per layer inside a CUDA graph."""
    import torch

    w, dev, bf, is_prompt = size["width"], x.device, x.dtype, rows == prompt_len
    seqs, n_seqs = (ctx.seq_slot, ctx.seq_q_start, ctx.seq_q_len), ctx.n_seqs
    # (a stream a call: together more than L2 holds at the prompt's size)
    streams = [torch.randn(rows, w, device=dev) for _ in blocks]
    y, z = rnd(rows, w), rnd(rows, w)
    us = in_graph([lambda b=b, s=s: ops.residual_norm(s, bf, 1e-6, (y, None, None, 0.0, z), b.norm1.weight)
                   for b, s in zip(blocks, streams)])
    out[f"{name}: two outputs + residual sum + norm"] = bw(us, rows * w * (4 + 4 + 2 + 2 + 2))
    table = rnd(spec.vocab_size, w)
    us = in_graph([lambda s=s: ops.residual_join(s, (y, None, None, 0.0, z), ctx.tokens, table) for s in streams])
    out[f"{name}: stream and embedding side by side"] = bw(us, rows * w * (4 + 2 + 2 + 2 + 4))
    joined, weights = rnd(rows, 2 * w), [rnd(w, 2 * w) for _ in range(8)]
    us = in_graph([lambda m=m: ops.linear(joined, m, out_float=True) for m in weights])
    out[f"{name}: projection back to the stream"] = tc(us, rows * 4 * w * w) if is_prompt else bw(us, 4 * w * w)

    def of(kind):
        return [(b.mixer, e.cache) for b, e in zip(blocks, spec.schedule) if b.mixer.spec.kind == kind]

    pairs = of("gated_linear_attention")
    m = pairs[0][0]
    sp = m.spec
    proj = rnd(rows, m.stacked.shape[0])
    gate_at = 2 * m.qk + m.inner
    us = in_graph([lambda p=p: ops.low_rank_decay(proj, gate_at + m.inner, p.a2, p.a2_bias, sp.tau) for p, _ in pairs])
    out[f"{name}: decays of low rank"] = bw(us, rows * (m.qk * 4 + sp.decay_rank * 2))
    decay = ops.low_rank_decay(proj, gate_at + m.inner, m.a2, m.a2_bias, sp.tau)
    us = in_graph([lambda p=p, e=e: ops.state_scan("channel_decay", (proj, 0), (proj, m.qk), (proj, 2 * m.qk), None, None, None, None,
                                                    None, cache.entry_state(e), p.state_at, *seqs, sp.num_heads, sp.num_heads,
                                                    sp.head_dim, sp.value_dim, decay=decay) for p, e in pairs])
    d = bw(us, rows * (m.qk * 8 + m.inner * 6) + n_seqs * sp.num_heads * sp.head_dim * sp.value_dim * 4 * 2)
    d["gflops"] = rows * sp.num_heads * sp.head_dim * sp.value_dim * 5 / us / 1e3
    out[f"{name}: recurrence with a decay per channel (state walk)"] = d
    o32 = torch.randn(rows, m.inner, device=dev)
    us = in_graph([lambda p=p: ops.group_norm_gate(o32, proj, gate_at, p.gain, sp.num_heads, 1e-6, False, bf) for p, _ in pairs])
    out[f"{name}: head norm + gate"] = bw(us, rows * m.inner * (4 + 2 + 2))

    pairs = of("sink_attention")
    a = pairs[0][0]
    sp = a.spec
    heads, kvh, dim, vdim = sp.num_heads, sp.num_kv_heads, sp.head_dim, sp.value_dim
    proj = rnd(rows, a.qkvg.shape[0])
    us = in_graph([lambda p=p, e=e: ops.short_conv(proj, 0, a.convolved, p.taps, None, p.biases, cache.entry_state(e), p.state_at,
                                                    *seqs, ctx.max_q_len) for p, e in pairs])
    out[f"{name}: bias + short convolution ({a.convolved} channels)"] = bw(us, rows * a.convolved * 4 + n_seqs * (sp.conv - 1) * a.convolved * 8)

    def prepare(p, e):
        k, v = cache.entry_pages(e)
        ops.sink_prepare_norm(proj, heads, kvh, dim, vdim, ctx.tok_pos, ctx.tok_slot, cache.block_table, k, v, a.position.rotation(),
                              p.row_norm, False, sp.norm_eps)

    def attend(p, e, sink):
        k, v = cache.entry_pages(e)
        return ops.sink_attention_step(proj, k, v, cache.block_table, ctx, heads, kvh, dim, vdim, sp.scale, None, sink, None, None,
                                       sp.window, 0, sp.softcap)

    us = in_graph([lambda p=p, e=e: prepare(p, e) for p, e in pairs])
    out[f"{name}: row norms, rotation, cache write"] = bw(us, rows * 2 * (2 * heads * dim + 2 * kvh * (dim + vdim)))
    seen = lambda p: min(p + 1, sp.window)  # noqa: E731
    for title, with_sink in (("window, cap, sink: attention", True), ("window, cap, no sink: attention", False)):
        us = in_graph([lambda p=p, e=e: attend(p, e, p.sink if with_sink else None) for p, e in pairs])
        out[f"{name}: {title}"] = (tc(us, heads * 2 * (dim + vdim) * sum(seen(p) for p in range(prompt_len))) if is_prompt
                                   else bw(us, batch * seen(context) * kvh * (dim + vdim) * 2))

    pairs = of("latent_attention")
    m = pairs[0][0]
    sp = m.spec
    proj = rnd(rows, m.down.shape[0])
    cos, sin = ops.latent_tables(m.position.rotation(), sp.position.dims)
    us = in_graph([lambda p=p, e=e: ops.latent_prepare(proj, p.q_gain, p.kv_gain, 1e-6, cos, sin, ctx.tok_pos, ctx.tok_slot,
                                                        cache.block_table, cache.entry_pages(e)[0], sp.q_rank, sp.kv_rank, sp.rot_dim,
                                                        sp.position.dims, kv_col=m.kv_at) for p, e in pairs])
    out[f"{name}: latent norms, rotation, cache write"] = bw(us, rows * 2 * 2 * (sp.q_rank + m.row))
    qa = rnd(rows, sp.num_heads, m.row)
    forms = [("latent attention, sink", None, True), ("latent attention, no sink", None, False)]
    forms += [("latent attention, window of 1,024, no sink (Kesedra's form)", 1024, False)]
    for title, window, with_sink in forms:
        us = in_graph([lambda p=p, e=e: ops.latent_attention_step(qa, cache.entry_pages(e)[0], cache.block_table, ctx, sp.num_heads,
                                                                   sp.kv_rank, sp.rot_dim, sp.scale, window, p.sink if with_sink else None)
                       for p, e in pairs])
        span = lambda p: min(p + 1, window or p + 1)  # noqa: E731
        out[f"{name}: {title}"] = (tc(us, sp.num_heads * 2 * (m.row + sp.kv_rank) * sum(span(p) for p in range(prompt_len))) if is_prompt
                                   else bw(us, batch * span(context) * m.row * 2))
    heads_out = rnd(rows, m.gate_size)
    us = in_graph([lambda p=p: ops.sigmoid_gate(heads_out, proj, sp.q_rank) for p, _ in pairs])
    out[f"{name}: output gate"] = bw(us, rows * m.gate_size * 2 * 3)
    ff = [b.feed_forward for b in blocks]
    us = in_graph([lambda f=f: f(x, None) for f in ff])
    inner = ff[0].spec.intermediate_size
    out[f"{name}: feed-forward (gate, up, down)"] = tc(us, rows * 6 * inner * w) if is_prompt else bw(us, 6 * inner * w)


def salulorn_compare(args) -> int:
    """Beside Setotar: the closest design this library has (window attention with biases, convolutions and capped scores,
    row norms, a recurrence with a matrix state per head, a 32-bit residual); the latent attention is also timed in the
    form it has in Kesedra."""
    if args.layers_given and args.layers < 5:
        raise SystemExit("this comparison needs 5 layers or more: three kinds, two of them run twice")
    return compare_with_qwen3(args, "salulorn", "Salulorn", salulorn_config, salulorn_kernels_alone, ["2048"],
                              beside=("setotar", "Setotar", setotar_config, setotar_kernels_alone))


def kesedra_compare(args) -> int:
    # the 2048 size alone by default: at 2560 with 8 layers a prompt step of this design failed to return while
    # its kernels still released their successors early; the larger sizes have not been timed since and run
    # when they are named
    return compare_with_qwen3(args, "kesedra", "Kesedra", kesedra_config, kesedra_kernels_alone, ["2048"])


def korurax_compare(args) -> int:
    return compare_with_qwen3(args, "korurax", "Korurax", korurax_config, korurax_kernels_alone, list(DESIGN_SIZES))


def compare_with_qwen3(args, design_key, design_title, config_of, own_kernels, default_sizes, beside=None) -> int:
    """``--design kesedra`` / ``korurax`` / ``bavedra`` / ``setotar`` / ``salulorn``: prefill and decode throughput of that design beside Qwen3
    (or, with ``beside = (key, title, config_of, kernels_alone)``, beside that design: the closest model this library
    has) at equal width, dense feed-forward, vocabulary and head count, and the design's own kernels alone beside the
    other's like kernels, each against its roofline.  Every number is timed on the device with CUDA events; the
    kernels alone run inside a CUDA graph, once per layer.  Prints one JSON line."""
    other_key, other_title, other_config, other_kernels = beside or ("qwen3", "Qwen3", qwen3_config, qwen3_kernels_alone)
    kernels_of = {design_key: own_kernels, other_key: other_kernels}
    import torch

    from starter_b200 import ops
    from starter_b200.config import config_from_dict
    from starter_b200.engine import ModelRunner, StepEntry, random_model

    pk = peaks()
    layers = args.layers if args.layers_given else 8
    batch, context, prompt_len = args.batch, 2048, PROMPT
    warmup, steps = max(args.warmup, 3), max(min(args.steps, 64), 1)
    sampler = ClockSampler()
    sampler.start()
    windows = []
    gen = torch.Generator().manual_seed(0)
    dev = torch.device("cuda:0")
    bf = torch.bfloat16

    def timed(fn, reps):
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        t0 = time.monotonic()
        start.record()
        for _ in range(reps):
            fn()
        stop.record()
        torch.cuda.synchronize()
        windows.append((t0, time.monotonic()))
        return start.elapsed_time(stop) / reps

    def in_graph(calls):
        """Microseconds per call of ``calls`` (one per layer), captured together and replayed."""
        for c in calls:
            c()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for c in calls:
                c()
        graph.replay()
        return timed(graph.replay, 5) / len(calls) * 1e3

    def rnd(*shape):
        return (torch.randn(*shape, device=dev) * 0.5).to(bf)

    def say(*what):
        torch.cuda.synchronize()
        print("[bench]", *what, file=sys.stderr, flush=True)

    def bw(us, moved):
        return dict(us=us, gbs=moved / us / 1e3, frac_of_copy_peak=moved / us / 1e3 / pk["hbm_gbs"])

    def tc(us, flops):
        return dict(us=us, tflops=flops / us / 1e6, frac_of_bf16_peak=flops / us / 1e6 / pk["bf16_tflops"])

    def kernels_alone(model, runner, design, size):
        spec = model.spec
        blocks = [model.blocks[e.layer] for e in spec.schedule]
        cache = runner.cache
        w = size["width"]
        out = {}
        slots = [runner.open_sequence() for _ in range(batch)]
        for s in slots:
            runner.step([StepEntry(s, torch.randint(0, spec.vocab_size, (context,), generator=gen).tolist(), [])])
        for rows, name in ((prompt_len, "prompt"), (batch, "decode")):
            if rows == prompt_len:
                slot = runner.open_sequence()
                ctx = runner.make_context([StepEntry(slot, [1] * prompt_len, [])])
            else:
                ctx = runner.make_context([StepEntry(s, [1], []) for s in slots])
            x = rnd(rows, w)
            say(design, name, "kernels alone")
            kernels_of[design](ops, out, name, rows, x, blocks, spec, cache, ctx, size, batch, context, prompt_len, rnd,
                               in_graph, bw, tc)
            if rows == prompt_len:
                runner.close_sequence(slot)
            else:
                for slot_, length in zip(ctx.host["seq_slot"].tolist(), ctx.host["seq_kv_len"].tolist()):
                    cache.lengths[slot_] = length - 1       # the context made above counted a token that no step ran
        for s in slots:
            runner.close_sequence(s)
        return {k: {a: round(b, 4 if "frac" in a else 1) for a, b in v.items()} for k, v in out.items()}

    results = {}
    for size_name in (args.design_sizes.split(",") if args.design_sizes else default_sizes):
        size = DESIGN_SIZES[size_name]
        row = {"layers": layers}
        for design, raw in ((design_key, config_of(size, layers)), (other_key, other_config(size, layers))):
            config = config_from_dict(raw)
            model = random_model(config, seed=0, dtype="bfloat16")
            vocab = model.spec.vocab_size
            runner = ModelRunner(model, max_tokens=(batch + 1) * (context + 256) + prompt_len, max_sequences=batch + 2)
            prompt = torch.randint(0, vocab, (prompt_len,), generator=gen).tolist()

            def prefill_once():
                slot = runner.open_sequence()
                runner.step([StepEntry(slot, prompt, [prompt_len - 1])])
                runner.close_sequence(slot)

            say(size_name, design, "model built")
            for _ in range(warmup):
                prefill_once()
                say("one prompt step done")
            prefill_ms = timed(prefill_once, 5)
            say("prompt", round(prefill_ms, 3), "ms")
            slots = [runner.open_sequence() for _ in range(batch)]
            for s in slots:
                runner.reserve(s, context + 256)
                runner.step([StepEntry(s, torch.randint(0, vocab, (context,), generator=gen).tolist(), [])])
            entries = [StepEntry(s, [1], [0]) for s in slots]

            def one():
                runner.decode_tokens(entries, [0.0] * batch, [0] * batch)

            for _ in range(warmup):
                one()
            decode_ms = timed(one, steps)
            say("single-token step", round(decode_ms, 4), "ms")
            for s in slots:
                runner.close_sequence(s)
            runner.check_status()
            row[design] = {
                "prefill_tok_s": round(prompt_len / prefill_ms * 1e3, 1), "prefill_ms": round(prefill_ms, 3),
                "decode_tok_s": round(batch / decode_ms * 1e3, 1), "decode_ms_per_step": round(decode_ms, 4),
                "weight_mb_per_step": round(model.step_weight_bytes() / 1e6, 1),
                "kernels_per_decode_step": runner.graphs.kernels_per_replay.get(batch),
                "kernels": kernels_alone(model, runner, design, size),
            }
            del runner, model
            torch.cuda.empty_cache()
        results[size_name] = row
    print(json.dumps({
        "metric": "prefill tok/s at 2,048 tokens and decode tok/s at batch %d, context 2,048: %s beside %s at "
                  "equal sizes (BF16, random weights)" % (batch, design_title, other_title),
        "unit": "tok/s", "n_gpus": 1, "dtype": "bf16", "steps": steps, "warmup": warmup,
        "data": "synthetic: random weights, uniform random token ids", "peaks": pk,
        "sizes": {k: DESIGN_SIZES[k] for k in results}, "results": results, "clocks": sampler.stop(windows)}))
    return 0


def main() -> int:
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=256)
    parser.add_argument("--warmup", type=int, default=5)
    parser.add_argument("--impl", default="ours", choices=["ours", "reference"])
    parser.add_argument("--layers", type=int, default=QWEN3_4B["num_hidden_layers"],
                        help="fewer layers than the model has (both numbers are reported)")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--skip-points", action="store_true", help="leave out batch 1 and 64")
    parser.add_argument("--workload", choices=sorted(WORKLOADS), default=None,
                        help="instead of the default run: one of the further rows (other model sizes)")
    parser.add_argument("--decode-at", type=int, default=DECODE_AT,
                        help="cached tokens per sequence at which decode is timed (default: the middle of the "
                             "generation range); the cache is sized for it")
    parser.add_argument("--per-stage", action="store_true",
                        help="also print where a decode step's time goes, kernel by kernel (stderr)")
    parser.add_argument("--design", choices=["goguvik", "kesedra", "korurax", "bavedra", "setotar", "salulorn"], default=None,
                        help="instead of the default run: that design beside Qwen3 (Bavedra: Kesedra; Setotar: Bavedra; Salulorn: Setotar) at equal "
                             "sizes (prefill, decode, and each design's own kernels against their rooflines)")
    parser.add_argument("--design-sizes", default=None, help="comma-separated subset of " + ",".join(DESIGN_SIZES))
    args = parser.parse_args()
    args.layers_given = "--layers" in sys.argv
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this library has no multi-GPU path (asked for {args.gpus})")
        return 2
    if args.impl == "reference":
        return reference_arm(args)
    if args.workload:
        return workload(args)
    if args.design == "korurax":
        return korurax_compare(args)
    if args.design == "salulorn":
        return salulorn_compare(args)
    if args.design == "setotar":
        return setotar_compare(args)
    if args.design == "bavedra":
        return bavedra_compare(args)
    if args.design == "kesedra":
        return kesedra_compare(args)
    if args.design:
        return design_compare(args)
    warmup = max(args.warmup, 3)
    steps = max(args.steps, 1)
    decode_at = args.decode_at
    context = max(CONTEXT, -(-(decode_at + warmup + 2 * steps + 2) // 64) * 64)     # whole cache pages

    import torch

    from starter_b200 import ops
    from starter_b200.config import config_from_dict
    from starter_b200.engine import ModelRunner, StepEntry, random_model
    from starter_b200.engine.entry import Engine

    raw = dict(QWEN3_4B, num_hidden_layers=args.layers)
    config = config_from_dict(raw)
    model = random_model(config, seed=0, dtype="bfloat16")
    vocab = config.vocab_size
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    windows = []
    gen = torch.Generator().manual_seed(0)

    def prompt(n):
        return torch.randint(0, vocab, (n,), generator=gen).tolist()

    max_batch = max(args.batch, 1 if args.skip_points else 64)
    runner = ModelRunner(model, max_tokens=max_batch * context, max_sequences=max_batch)

    def timed(fn, reps):
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        t0 = time.monotonic()
        start.record()
        for _ in range(reps):
            fn()
        stop.record()
        torch.cuda.synchronize()
        windows.append((t0, time.monotonic()))
        return start.elapsed_time(stop) / reps

    # ---------------------------------------------------------------- prefill of 2,048 tokens
    def prefill_once():
        slot = runner.open_sequence()
        runner.step([StepEntry(slot, prefill_prompt, [PROMPT - 1])])
        runner.close_sequence(slot)

    prefill_prompt = prompt(PROMPT)
    for _ in range(warmup):
        prefill_once()
    prefill_ms = timed(prefill_once, 5)
    h, nh, kv, d, inter, layers = (config.hidden_size, config.num_attention_heads,
                                   config.num_key_value_heads, config.head_dim,
                                   config.intermediate_size, args.layers)
    per_token = 2 * h * (nh + 2 * kv) * d + 2 * nh * d * h + 2 * h * 2 * inter + 2 * inter * h
    attn = 4 * nh * d * PROMPT * (PROMPT + 1) / 2
    prefill_flops = layers * (per_token * PROMPT + attn) + 2 * h * vocab
    prefill = {"value": round(PROMPT / prefill_ms * 1e3, 1), "tokens": PROMPT, "ms": round(prefill_ms, 3),
               "frac": round(prefill_flops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4),
               # the same against the vendor GEMM's throughput in a seconds-long loop under the power
               # cap: the prompt step is timed over several back-to-back repetitions
               "frac_of_sustained": round(prefill_flops / (prefill_ms * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 4)}

    # ---------------------------------------------------------------- decode, device-timed
    def decode_point(batch):
        slots = [runner.open_sequence() for _ in range(batch)]
        for s in slots:
            runner.reserve(s, context)
            runner.step([StepEntry(s, prompt(decode_at), [])])
        entries = [StepEntry(s, [1], [0]) for s in slots]
        zeros = [0.0] * batch
        keys = [0] * batch

        def one():
            runner.decode_tokens(entries, zeros, keys)

        for _ in range(warmup):
            one()
        if args.per_stage:
            per_layer_us = per_stage(model, runner, slots, batch, pk["hbm_gbs"])
            one()
        before = ops.launch_count
        captured = len(runner.graphs.graphs)
        ms = timed(one, steps)
        if len(runner.graphs.graphs) != captured:
            # the sequences grew into the next length class inside the timed steps and its graph was
            # captured there: that is set-up, not a decode step; time the same number of steps again
            before = ops.launch_count
            ms = timed(one, steps)
        if args.per_stage:
            print(f"  the whole step: {ms * 1e3:.1f} us = {len(model.spec.schedule)} layers x "
                  f"{(ms * 1e3) / len(model.spec.schedule):.1f} us (head, sampling and embedding included); "
                  f"launched one by one the layers' kernels add up to {per_layer_us:.1f} us a layer",
                  file=sys.stderr)
        per_graph = runner.graphs.kernels_per_replay.get(batch, 0)
        launches = steps * per_graph + (ops.launch_count - before)
        for s in slots:
            runner.close_sequence(s)
        kv_bytes = runner.cache.bytes_per_token() * batch * (decode_at + warmup + steps / 2)
        return ms, launches, model.step_weight_bytes() + kv_bytes

    ms, launches, step_bytes = decode_point(args.batch)
    value = args.batch / ms * 1e3
    achieved = step_bytes / (ms * 1e-3) / 1e9
    points = {}
    if not args.skip_points:
        for b in (1, 64):
            b_ms, _, _ = decode_point(b)
            points[f"decode_b{b}"] = round(b / b_ms * 1e3, 1)

    # ---------------------------------------------------------------- end to end through Engine.generate
    del runner
    torch.cuda.empty_cache()

    def e2e_point(batch):
        """tok/s through the public call: prompts in as host lists, one list of ids out per step."""
        engine = Engine.from_model(model, max_batch=batch)
        stream = engine.generate([prompt(decode_at) for _ in range(batch)], warmup + steps + 2)
        next(stream)
        # every step's host-owned inputs (positions, slots, lengths, sampling settings) travel from
        # pinned host memory to the device and the drawn ids travel back to the host; the ids a step
        # consumes are the ones the step before drew on the device, so the loop launches a step
        # before it reads the one before (one step of lookahead, as the reference's loop does)
        engine.runner.self_feeding = False
        for _ in range(warmup):
            next(stream)
        torch.cuda.synchronize()
        t0 = time.monotonic()
        for _ in range(steps):
            next(stream)
        torch.cuda.synchronize()
        t1 = time.monotonic()
        windows.append((t0, t1))
        stream.close()
        engine.runner.check_status()
        del engine
        torch.cuda.empty_cache()
        return batch * steps / (t1 - t0)

    e2e_value = e2e_point(args.batch)
    if not args.skip_points:
        points["e2e_b1"] = round(e2e_point(1), 1)

    clocks = sampler.stop(windows)
    line = {
        "metric": METRIC,
        "value": round(value, 1), "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: random weights N(0,0.02), uniform random token ids",
        "config": dict(config_block(args.layers, args.batch, pk["source"]), decode_context=decode_at),
        "e2e": {"value": round(e2e_value, 1), "unit": "tok/s", "h2d_bytes_per_step": 5 * 4 * args.batch,
                "d2h_bytes_per_step": 4 * args.batch},
        "gpu_launches": launches,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
        "clocks": clocks,
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
