#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at LFM2-1.2B sizes with random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--context 4096] [--layers N] [--dtype bfloat16|float32]

One JSON line on stdout.  ``value`` is decoded tokens per second at the given batch, device-
timed with CUDA events over regions of exactly K decode steps (each step: the packed index data
goes host->device, the captured decode graph replays, greedy tokens are chosen on the device).
The region is repeated, each time over the same positions of the same requests, until at least
0.3 s of device time has been measured, and the median region is reported, so that a small K
still gives a steady figure.  ``e2e`` is the same metric through the engine loop a user drives
(scheduler, step, sampler, host tokens in and out, wall clock).  ``prefill`` times one
2,048-token prompt in one step; ``roofline`` relates the decode step to the bytes it must read;
``kernels`` says where the decode step's and the prefill's time goes, kernel family by kernel
family, each against the measured peak that bounds it; ``points`` holds decode at batch 1 and 64
and the true 32-bit path's figures.  Peaks come from MEASURED_PEAKS.json when the file is there,
else from the fallback figures.

The engine runs on one GPU: with --gpus above 1 it says so and exits with 2.
"""
import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

# LFM2-1.2B layer sizes: full_attention at layers 2, 5, 8, 10, 12, 14 of 16
LFM2_1P2B = {
    "architectures": ["Lfm2ForCausalLM"], "model_type": "lfm2",
    "vocab_size": 65536, "hidden_size": 2048, "intermediate_size": 12288,
    "block_auto_adjust_ff_dim": True, "block_ffn_dim_multiplier": 1.0, "block_multiple_of": 256,
    "num_hidden_layers": 16, "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 64,
    "conv_L_cache": 3, "conv_bias": False, "rope_theta": 1000000.0, "norm_eps": 1e-5,
    "tie_word_embeddings": True, "max_position_embeddings": 128000,
    "layer_types": ["full_attention" if l in (2, 5, 8, 10, 12, 14) else "conv" for l in range(16)],
}


def lfm2_sizes(name):
    """The other two sizes the benchmark configurations name (random weights, so only the layer
    sizes matter).  The 2.6B stack has 8 attention layers among 30; they are spread evenly here."""
    cfg = dict(LFM2_1P2B)
    if name == "1.2b":
        return cfg
    if name == "700m":
        cfg.update(hidden_size=1536, intermediate_size=10240, num_attention_heads=24)
        return cfg
    if name == "2.6b":
        attn = (2, 6, 10, 14, 18, 21, 24, 27)
        cfg.update(intermediate_size=10752, num_hidden_layers=30,
                   layer_types=["full_attention" if l in attn else "conv" for l in range(30)])
        return cfg
    raise ValueError(name)


def peaks():
    p = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                m = json.load(f)
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                if isinstance(m.get(k), (int, float)):
                    p[k] = float(m[k])
            p["source"] = "measured"
        except (OSError, ValueError):
            pass
    return p


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "50"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
        sm = sorted(int(r[0]) for r in self.rows if len(r) >= 6 and r[0].isdigit())
        mx = [int(r[1]) for r in self.rows if len(r) >= 6 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({n for r in self.rows if len(r) >= 6 for n, v in zip(names, r[2:6]) if v.lower().startswith("active")})
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(sm)}


def part_tensors(plan):
    """(label, tensor) for every tensor that a part of the plan holds, each tensor once; the label is
    the part's class and attribute name, e.g. ``SwiGLU.w_gate_up``.  Walks whatever parts the
    blocks are made of, so a plan of other parts needs no change here."""
    import torch
    from vapi_b200.parts.base import Part
    seen = set()

    def members(v):
        """A part's attribute, or what a list or dictionary in it holds."""
        if isinstance(v, (list, tuple)):
            for x in v:
                yield from members(x)
        elif isinstance(v, dict):
            for x in v.values():
                yield from members(x)
        else:
            yield v

    def of_part(part):
        for name, held in vars(part).items():
            for v in members(held):
                if isinstance(v, torch.Tensor) and v.data_ptr() not in seen:
                    seen.add(v.data_ptr())
                    yield f"{type(part).__name__}.{name}", v
        for held in vars(part).values():
            for v in members(held):
                if isinstance(v, Part):
                    yield from of_part(v)

    for call in plan.order:
        yield from of_part(plan.layers[call.layer])
    for part in getattr(plan, "stream_parts", {}).values():
        yield from of_part(part)
    yield from of_part(plan.final_norm)
    yield from of_part(plan.head)        # tied: the embedding table, read once by the head
    yield from of_part(plan.embedding)


def model_numbers(runner):
    """Bytes of every weight a decode step reads once (the embedding table counts once: a step
    gathers a few rows of it and the tied head reads all of it), and matrix-product parameters."""
    wbytes, mm_params = 0, 0
    for label, t in part_tensors(runner.plan):
        if label in ("TokenEmbedding.table", "TokenEmbedding.bigram_table"):
            continue                      # (reached only when untied) a table is gathered from, not streamed
        wbytes += t.numel() * t.element_size()
        if t.dim() == 2 and t.shape[0] > 8:
            mm_params += t.numel()
    return wbytes, mm_params


def trace_table(events):
    """Rows for the last whole step among the stamps: the step's kernels in the order in which their
    dependency waits returned, each with how long it then took until the next kernel's wait returned
    (its own dependent work, its drain and the hand-over)."""
    rel = [e for e in events if e["kind"] == "released"]
    ends = [i for i, e in enumerate(rel) if e["library"] == "sampling"]
    if len(ends) < 2:
        return []
    step = rel[ends[-2] + 1:ends[-1] + 1]
    start = {}
    for e in events:
        if e["kind"] == "start":
            start.setdefault((e["library"], e["blocks"], e["threads"]), []).append(e["ns"])
    rows = []
    for a, b in zip(step, step[1:] + [None]):
        key = (a["library"], a["blocks"], a["threads"])
        began = max((t for t in start.get(key, []) if t <= a["ns"]), default=a["ns"])
        rows.append({"library": a["library"], "blocks": a["blocks"], "threads": a["threads"],
                     "waited_us": (a["ns"] - began) / 1e3, "at_us": (a["ns"] - step[0]["ns"]) / 1e3,
                     "until_next_us": (b["ns"] - a["ns"]) / 1e3 if b else None})
    return rows


#: the calls that are matrix products (time against the tensor peak); the rest move bytes
PRODUCTS = ("linear", "skinny_linear", "linear_tc", "prompt_linear", "skinny_shortconv")

#: the package's kernels as the parts call them, with the library each lives in
OPS = {"embed": "elementwise", "add_residual_ss": "elementwise", "resolve_tokens": "elementwise",
       "add_rmsnorm": "elementwise", "add_residual": "elementwise", "swiglu": "elementwise",
       "skinny_linear": "gemv", "skinny_shortconv": "gemv", "linear_tc": "linear_tc", "prompt_linear": "linear_prompt",
       "rope_cos_sin": "rope",
       "qk_norm_rope_write": "rope", "paged_attention": "attention", "decode_attention_fused": "attention",
       "shortconv": "shortconv", "sample_rows": "sampling", "sample_truncated": "sampling", "linear": "library",
       "postnorm_add_rmsnorm": "elementwise", "gated_group_rmsnorm": "elementwise", "scale_rows": "elementwise",
       "rope_cos_sin_scaled": "rope", "qk_norm_rope_write_split": "rope", "masked_attention": "attention_masked",
       "causal_conv_silu": "recurrent", "gated_delta": "recurrent", "state_space": "recurrent",
       "embed_sinusoid": "hyper", "hyper_read_norm": "hyper", "branch_rmsnorm_mean": "hyper", "sigmoid_gate": "hyper",
       "softcap": "hyper", "causal_conv": "recurrent", "rglru": "rglru", "relu_squared": "moe", "moe_route": "moe",
       "moe_experts": "moe", "matrix_memory": "linear_memory", "gated_linear_attention": "linear_memory",
       "fixed_decay_memory": "fixed_decay",
       "scaled_add_rmsnorm": "elementwise", "latent_prepare": "latent", "latent_rotate_q": "latent",
       "latent_attention": "attention_masked", "moe_table_route": "moe", "head_products": "library",
       "embed_bigram": "elementwise", "shift_add_rmsnorm": "elementwise", "xielu": "elementwise"}


class OpLog:
    """Stands between the parts and the kernels' Python faces for one measurement: every call is
    noted with the weight it streams (the first 2-D bfloat16/float32 matrix among its arguments
    that a part of the plan holds), the kernels it launched and, when ``events`` is set, CUDA
    events around it.  Calls made from inside another noted call are not noted again."""

    def __init__(self, ops, plan, events=False):
        import torch
        self.ops, self.torch, self.events = ops, torch, events
        self.labels = {t.data_ptr(): (label, t) for label, t in part_tensors(plan)}
        self.calls, self.depth, self.saved = [], 0, {}

    def __enter__(self):
        for name in OPS:
            fn = getattr(self.ops, name)
            self.saved[name] = fn
            setattr(self.ops, name, self._wrap(name, fn))
        return self

    def __exit__(self, *exc):
        for name, fn in self.saved.items():
            setattr(self.ops, name, fn)

    def _wrap(self, name, fn):
        torch = self.torch

        def call(*a, **kw):
            if self.depth:
                return fn(*a, **kw)
            self.depth += 1
            try:
                tensors = [t for t in list(a) + list(kw.values()) if isinstance(t, torch.Tensor)]
                weight = next((self.labels[t.data_ptr()] for t in tensors if t.data_ptr() in self.labels and t.dim() == 2), None)
                before = self.ops.launch_count
                ev = None
                if self.events:
                    ev = (torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True))
                    ev[0].record()
                out = fn(*a, **kw)
                if ev:
                    ev[1].record()
                outs = [t for t in (out if isinstance(out, tuple) else (out,)) if isinstance(t, torch.Tensor)]
                rows = max([t.shape[0] for t in outs if t.dim() >= 1] or [0])
                # what an elementwise call moves: its activations in and out (not the caches and states it
                # touches a few rows of, not the plan's own tensors)
                moved = sum(t.numel() * t.element_size() for t in tensors + outs
                            if t.dim() <= 3 and t.data_ptr() not in self.labels)
                if name == "embed":
                    moved *= 2            # the rows gathered from the table, and the stream written
                self.calls.append({"op": name, "weight": weight[0] if weight else None,
                                   "weight_shape": tuple(weight[1].shape) if weight else None,
                                   "weight_bytes": weight[1].numel() * weight[1].element_size() if weight else 0,
                                   "rows": rows, "moved_bytes": moved, "launches": self.ops.launch_count - before, "events": ev})
                return out
            finally:
                self.depth -= 1
        return call


def family_of(call):
    """The name under which a noted call is summed up: a product by the matrix it streams, any
    other kernel by its own name."""
    if call["op"] in PRODUCTS and call["weight"]:
        return call["weight"] + ("+conv" if call["op"] == "skinny_shortconv" else "")
    return call["op"]


def decode_kernel_table(args, pk, timeout=420):
    """Where the captured decode step's time goes: a second process runs a few steps of the same
    step with a measuring build of every kernel library (its kernels stamp the device clock) and
    names the kernels in launch order; this sums them up by family.  Each family's time is the time
    from the return of its kernels' dependency waits to the return of the next kernel's, so the
    families add up to the step; bytes are the weights and cache it has to read."""
    cmd = [sys.executable, os.path.abspath(__file__), "--only", "trace", "--rows-json", "--steps", "6", "--warmup", "4",
           "--batch", str(args.batch), "--context", str(args.context), "--sizes", args.sizes, "--layers", str(args.layers),
           "--page-size", str(args.page_size)]
    try:
        proc = subprocess.run(cmd, capture_output=True, text=True, timeout=timeout)
        line = next((l for l in proc.stdout.splitlines() if l.startswith('{"trace_rows"')), None)
        if proc.returncode != 0 or line is None:
            return {"unavailable": "the measuring pass failed: " + (proc.stderr.strip().splitlines() or ["no output"])[-1][:200]}
        rec = json.loads(line)
    except (subprocess.TimeoutExpired, OSError, ValueError) as e:
        return {"unavailable": f"the measuring pass failed: {type(e).__name__}"}
    if rec.get("mismatch"):
        return {"unavailable": rec["mismatch"]}
    fam = {}
    for r in rec["trace_rows"]:
        f = fam.setdefault(r["family"], {"us": 0.0, "bytes": 0, "launches": 0})
        f["us"] += r["us"] or 0.0
        f["bytes"] += r["bytes"]
        f["launches"] += 1
    out = {}
    for name, f in sorted(fam.items(), key=lambda kv: -kv[1]["us"]):
        gbs = f["bytes"] / (f["us"] * 1e-6) / 1e9 if f["us"] > 0 else 0.0
        out[name] = {"us": round(f["us"], 1), "launches": f["launches"], "MB": round(f["bytes"] / 1e6, 1),
                     "GBps": round(gbs, 0), "frac_hbm": round(gbs / pk["hbm_gbs"], 3)}
    return {"ms_per_step_with_stamps": rec["ms_per_step"], "families": out}


def run(args):
    if args.only == "trace":          # a measuring build of every kernel library, named before the first import
        os.environ["VAPI_NVCC_FLAGS"] = (os.environ.get("VAPI_NVCC_FLAGS", "") + " -DVAPI_TRACE").strip()
    import torch
    from vapi_b200 import ops
    from vapi_b200.engine.engine import Engine
    from vapi_b200.engine.runner import ModelRunner, parse_dtype
    from vapi_b200.engine.scheduler import SchedulerConfig
    from vapi_b200.engine.step import StepEntry
    from vapi_b200.sampling.params import SamplingParams

    pk = peaks()
    cfg = lfm2_sizes(args.sizes)
    full_layers = cfg["num_hidden_layers"]
    layers = args.layers or full_layers
    if args.only == "serve":
        return serve(args, cfg)
    if args.only == "mixers":
        return mixers(args)
    if layers != full_layers:
        cfg["num_hidden_layers"] = layers
        cfg["layer_types"] = cfg["layer_types"][:layers]
    ctx_len, B = args.context, args.batch
    dev = torch.device("cuda:0")
    torch.cuda.set_device(dev)
    max_b = max(B, 64)
    page = args.page_size or ModelRunner.default_page_size
    gen = torch.Generator().manual_seed(1)
    vocab = cfg["vocab_size"]
    MIN_TIMED_S = 0.3

    def make_runner(dtype, most_requests=max_b):
        n_pages = most_requests * (-(-(ctx_len + 256) // page)) + 8      # (the engine-loop run lets contexts grow past ctx_len)
        return ModelRunner.from_random(cfg, seed=0, dtype=dtype, device="cuda:0", num_pages=n_pages, page_size=page,
                                       max_requests=most_requests, max_batched_tokens=8192, max_context=ctx_len + 256,
                                       watermark=0.0, validate=False)

    def fill(runner, batch, length):
        """Open `batch` requests and prefill them to `length` tokens in portions (untimed)."""
        rcs = []
        for i in range(batch):
            rc = runner.cache.open(("bench", batch, i))
            toks = torch.randint(0, vocab, (length,), generator=gen).tolist()
            pos = 0
            while pos < length:
                q = min(4096, length - pos)
                assert runner.cache.reserve(rc, pos + q)
                runner.step([StepEntry(rc, toks[pos:pos + q], [])])
                pos += q
            rcs.append(rc)
        torch.cuda.synchronize()
        return rcs

    def decode_steps(runner, rcs, count, timed):
        """`count` decode steps on the stream; device time in ms when `timed`."""
        toks = torch.randint(0, vocab, (count, len(rcs)), generator=gen).tolist()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for s in range(count):
            entries = []
            for j, rc in enumerate(rcs):
                assert runner.cache.reserve(rc, rc.num_tokens + 1)
                entries.append(StepEntry(rc, [toks[s][j]], [0]))
            logits = runner.step_decode_graph(entries)
            if logits is None:
                logits = runner.step(entries)
            ops.sample_rows(logits)
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) if timed else 0.0

    def decode_point(runner, batch, steps, warmup, clocks=None, min_s=MIN_TIMED_S):
        """Regions of exactly `steps` decode steps that end at the context length, repeated until
        `min_s` seconds of device time are measured (three regions at least); every region decodes
        the same positions of the same requests again (the requests' counts of computed positions
        are set back in between, which leaves their pages in place).  Returns the median region."""
        start_len = ctx_len - steps - 1
        rcs = fill(runner, batch, start_len)

        def rewind():
            for rc in rcs:
                runner.cache.commit(rc, start_len)

        done = 0
        while done < warmup:
            k = min(steps, warmup - done)
            decode_steps(runner, rcs, k, False)
            rewind()
            done += k
        if clocks:
            clocks.start()
        regions, total, launches = [], 0.0, 0
        while len(regions) < 3 or (total < min_s * 1e3 and len(regions) < 400):
            before = ops.launch_count
            ms = decode_steps(runner, rcs, steps, True)
            launches = ops.launch_count - before
            kv_bytes = sum(rc.num_tokens for rc in rcs) * runner.cache.bytes_per_token() + \
                batch * runner.cache.state_bytes_per_request()
            rewind()
            regions.append(ms)
            total += ms
        clk = clocks.stop() if clocks else None
        for rc in rcs:
            runner.cache.close(rc)
        ms = sorted(regions)[len(regions) // 2]
        return ms, launches, clk, kv_bytes, len(regions)

    if args.only == "trace":
        return trace_pass(args, make_runner(args.dtype), fill, decode_steps, ops, ctx_len, B)
    dtype = "float32" if parse_dtype(args.dtype) == torch.float32 else "bfloat16"
    runner = make_runner(dtype)
    wbytes, mm_params = model_numbers(runner)
    fp32_peak = measure_fp32_peak(dev) if (dtype == "float32" or args.only == "all") else None
    peak_tflops = fp32_peak if dtype == "float32" else pk["bf16_tflops"]
    if args.only == "prefill":
        p, fam = measure_prefill(runner, ops, mm_params, pk, peak_tflops, gen, vocab, dev, warm=max(1, min(args.warmup, 3)),
                                 iters=max(1, min(args.steps, 5)))
        print(json.dumps({"only": "prefill", "dtype": dtype, "prefill": p, "kernels": fam}), flush=True)
        return 0
    # ---- headline: decode at the given batch -----------------------------------------
    clocks = ClockSampler()
    ms, launches, clk, kv_bytes, regions = decode_point(runner, B, args.steps, args.warmup, clocks)
    ms_step = ms / args.steps
    value = B * args.steps / (ms / 1e3)
    print(f"[bench] decode b{B} {dtype}: {value:.0f} tok/s, {ms_step:.4f} ms/step (median of {regions} regions of "
          f"{args.steps} steps)", file=sys.stderr, flush=True)
    step_bytes = wbytes + kv_bytes
    achieved = step_bytes / (ms_step / 1e3) / 1e9

    if args.only == "decode":
        print(json.dumps({"only": "decode", "dtype": dtype, "value": round(value, 1), "ms_per_step": round(ms_step, 4),
                          "gpu_launches": launches, "roofline_frac": round(achieved / pk["hbm_gbs"], 4)}), flush=True)
        return 0
    # ---- other batch sizes ----------------------------------------------------------
    points = {}
    for b in (1, 64):
        m, _, _, kvb, _ = decode_point(runner, b, args.steps, max(8, args.warmup))
        points[f"decode_b{b}"] = round(b * args.steps / (m / 1e3), 1)
        points[f"decode_b{b}_frac_hbm"] = round((wbytes + kvb) / (m / args.steps / 1e3) / 1e9 / pk["hbm_gbs"], 4)
        print(f"[bench] decode b{b} {dtype}: {points[f'decode_b{b}']} tok/s, {m / args.steps:.4f} ms/step, "
              f"{points[f'decode_b{b}_frac_hbm']} of the HBM peak", file=sys.stderr, flush=True)

    prefill, prefill_families = measure_prefill(runner, ops, mm_params, pk, peak_tflops, gen, vocab, dev)
    c = runner.plan.config
    n_attn = len(runner.cache.paged[0].sites) if runner.cache.paged else 0

    # ---- end to end through the engine loop ----------------------------------------
    # regions of `steps` engine steps, one after the other (the contexts grow): as many as 0.3 s needs, and no
    # more than keep every request below the context limit with the middle region near the context length
    warm_e2e = max(8, args.warmup)
    reps = max(1, min(int(MIN_TIMED_S * 1e3 / max(ms, 1e-3)) + 1, (512 + args.steps - 40 - warm_e2e) // args.steps))
    eng = Engine(runner, SchedulerConfig(max_concurrent_seqs=max_b, max_batched_tokens=8192,
                                         prefill_chunk_tokens=4096, max_context=ctx_len + 256), use_graphs=True)
    # the middle region ends near the context length; requests finish their prompts at different
    # steps, so leave room for the early ones
    start_len = max(16, ctx_len - warm_e2e - (reps * args.steps) // 2 - args.steps // 2 - 2)
    for i in range(B):
        prompt = torch.randint(0, vocab, (start_len,), generator=gen).tolist()
        eng.admit(("e2e", i), prompt, SamplingParams(temperature=0.0, max_tokens=warm_e2e + reps * args.steps + 128,
                                                     ignore_eos=True))
    while any(s.needs_prefill() for s in eng.scheduler.seqs.values()) or eng.scheduler.num_waiting:
        eng.step()
    for _ in range(warm_e2e):
        eng.step()
    torch.cuda.synchronize()
    st0 = dict(eng.stats.__dict__)
    e2e_regions, h2d, d2h = [], 0, 0
    for _ in range(reps):
        t0 = time.perf_counter()
        got = 0
        for _ in range(args.steps):
            out = eng.step()        # (the engine runs one step ahead: these are the tokens of the step before)
            got += len(out.new_tokens)
            h2d += runner.packer.h2d_bytes_last + eng.sampler.h2d_bytes_last
            d2h += eng.sampler.d2h_bytes_last
        torch.cuda.synchronize()
        e2e_regions.append(time.perf_counter() - t0)
        assert got == B * args.steps, (got, eng.stats, eng.last_error)
    e2e_s = sorted(e2e_regions)[len(e2e_regions) // 2]
    e2e = {"value": round(B * args.steps / e2e_s, 1), "unit": "tokens/s",
           "h2d_bytes_per_step": h2d // (reps * args.steps), "d2h_bytes_per_step": d2h // (reps * args.steps),
           "ms_per_step": round(e2e_s * 1e3 / args.steps, 4), "regions": reps}
    runner.check_status()
    st, n = eng.stats, reps * args.steps
    host = {k: round((getattr(st, k) - st0[k]) / n, 4) for k in ("schedule_ms", "forward_ms", "sample_ms", "commit_ms")}
    e2e["host_ms_per_decode_step"] = host
    print(f"[bench] e2e: {e2e}", file=sys.stderr, flush=True)
    for seq in list(eng.scheduler.seqs.values()):
        eng.cancel(seq.seq_id)
    eng.run()

    # ---- the true 32-bit path (the default run is bfloat16) -----------------------------
    if dtype == "bfloat16" and args.only == "all" and not args.no_fp32:
        del eng, runner
        torch.cuda.empty_cache()
        r32 = make_runner("float32", most_requests=max(B, 8))
        w32, mm32 = model_numbers(r32)
        for b in sorted({1, B}):
            m, _, _, kvb, _ = decode_point(r32, b, args.steps, max(8, args.warmup))
            points[f"decode_b{b}_fp32"] = round(b * args.steps / (m / 1e3), 1)
            points[f"decode_b{b}_fp32_frac_hbm"] = round((w32 + kvb) / (m / args.steps / 1e3) / 1e9 / pk["hbm_gbs"], 4)
        p32, _ = measure_prefill(r32, ops, mm32, pk, fp32_peak, gen, vocab, dev, warm=2, iters=3, families=False)
        points["prefill_fp32"] = p32["value"]
        points["prefill_fp32_ms"] = p32["ms"]
        points["prefill_fp32_frac"] = p32["frac"]
        print(f"[bench] float32: {({k: v for k, v in points.items() if 'fp32' in k})}", file=sys.stderr, flush=True)
        del r32
        torch.cuda.empty_cache()

    kernels = {"prefill": prefill_families}
    if dtype == "bfloat16" and not args.no_kernels:
        kernels[f"decode_b{B}"] = decode_kernel_table(args, pk)

    line = {
        "metric": "LFM2-%s decode tokens/s (batch %d, context %d), random weights" % (args.sizes.upper(), B, ctx_len),
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms_step, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16" if dtype == "bfloat16" else "fp32",
        "data": "synthetic (seeded uniform-random token ids, random-init weights N(0, 0.02))",
        "impl": "vapi_b200",
        "config": {
            "model": "LFM2-%s sizes" % args.sizes.upper(), "global_batch": B, "seq_len": ctx_len, "parallelism": "single GPU",
            "layers": layers, "layers_of_configuration": full_layers, "attention_layers": n_attn,
            "hidden_size": c.hidden_size, "intermediate_size": c.intermediate_size, "vocab_size": c.vocab_size,
            "heads": c.num_attention_heads, "kv_heads": c.num_key_value_heads, "head_dim": c.head_dim,
            "conv_L_cache": c.conv_L_cache, "page_size": page, "cuda_graphs": True,
            "l2": "inputs larger than L2 (weights %.2f GB per step)" % (wbytes / 1e9),
            "peaks": pk["source"],
            "timing": "median of %d regions of %d steps over the same positions" % (regions, args.steps),
            "fp32_peak_tflops": fp32_peak,
        },
        "e2e": e2e,
        "gpu_launches": launches,
        "clocks": clk,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "bytes_per_step": int(step_bytes)},
        "points": points,
        "kernels": kernels,
    }
    print(json.dumps(line), flush=True)
    return 0


def trace_pass(args, runner, fill, decode_steps, ops, ctx_len, B):
    """A few decode steps of the measuring build: what one step's kernels did inside the captured
    graph, from their own time stamps; with --rows-json as one JSON line in which every kernel
    carries its family and the bytes it has to read."""
    import torch
    ops.trace_start()
    steps, warm = min(args.steps, 8), min(args.warmup, 4)
    rcs = fill(runner, B, ctx_len - steps - warm - 1)
    log = OpLog(ops, runner.plan)
    real_forward = runner.forward

    graph_calls = []

    def forward(ctx):               # the last forward pass before the steps is the one the graph holds
        log.calls.clear()
        out = real_forward(ctx)
        graph_calls[:] = list(log.calls)
        return out

    runner.forward = forward
    with log:
        decode_steps(runner, rcs, warm, False)
    runner.forward = real_forward
    ms = decode_steps(runner, rcs, steps, True)
    rows = trace_table(ops.trace_read())
    kv_per_site = sum(rc.num_tokens for rc in rcs) * runner.cache.bytes_per_token() / \
        max(1, sum(len(g.sites) for g in runner.cache.paged))
    state_per_site = B * runner.cache.state_bytes_per_request() / max(1, sum(len(g.sites) for g in runner.cache.state))
    if not args.rows_json:
        print(f"decode step, batch {B}, context {ctx_len}: {ms / steps:.4f} ms/step with the stamps on; one step's kernels in "
              f"the order in which their dependency waits returned", flush=True)
        print("   at us   library      blocks threads  waited us  until the next kernel's wait returns, us", flush=True)
        for r in rows:
            nxt = f"{r['until_next_us']:8.2f}" if r["until_next_us"] is not None else "       -"
            print(f"{r['at_us']:8.2f}   {r['library']:12s} {r['blocks']:6d} {r['threads']:7d}  {r['waited_us']:9.2f}  {nxt}", flush=True)
        return 0
    # name the stamped kernels: the graph's launches in order, then the sampler's
    expect = []
    for c in graph_calls:
        for k in range(c["launches"]):
            nbytes = (c["weight_bytes"] if c["op"] in PRODUCTS else c["moved_bytes"]) if k == 0 else 0
            if c["op"] in ("paged_attention", "decode_attention_fused") and k == 0:
                nbytes = int(kv_per_site)
            if c["op"] == "skinny_shortconv" and k == 0:
                nbytes += int(state_per_site)
            expect.append({"library": OPS[c["op"]], "family": family_of(c), "bytes": nbytes})
    expect.append({"library": "sampling", "family": "sample_rows", "bytes": B * runner.vocab_size * 4})
    out, mismatch = [], None
    if len(rows) != len(expect):
        mismatch = f"the step stamped {len(rows)} kernels where the launch log names {len(expect)}"
    else:
        for r, e in zip(rows, expect):
            if r["library"] != e["library"]:
                mismatch = f"a kernel of lib{r['library']} stands where the launch log names lib{e['library']}"
                break
            out.append({"family": e["family"], "bytes": e["bytes"], "us": r["until_next_us"], "blocks": r["blocks"]})
    print(json.dumps({"trace_rows": out, "mismatch": mismatch, "ms_per_step": round(ms / steps, 4)}), flush=True)
    return 0


def measure_fp32_peak(dev):
    """The library's float32 matrix product with every reduced-precision mode off, 4096^3, best of
    5 after 2 warm-ups, in TFLOP/s: the peak that the true 32-bit path's prefill is held against."""
    import torch
    from vapi_b200 import ops
    ops.strict_fp32()
    n = 4096
    a = torch.randn(n, n, device=dev)
    b = torch.randn(n, n, device=dev)
    best = None
    for it in range(7):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        torch.mm(a, b)
        e1.record()
        torch.cuda.synchronize()
        if it >= 2:
            t = e0.elapsed_time(e1)
            best = t if best is None else min(best, t)
    return round(2.0 * n ** 3 / (best / 1e3) / 1e12, 1)


def serve(args, cfg):
    """Continuous batching: --requests requests with random prompt lengths 128..2,048 arrive at
    once, each generates --max-tokens tokens (greedy); everything goes through the engine loop.
    One JSON line: generated tokens per second and all tokens (prompt + generated) per second."""
    import torch
    from vapi_b200.engine.engine import Engine
    from vapi_b200.engine.runner import ModelRunner
    from vapi_b200.engine.scheduler import SchedulerConfig
    from vapi_b200.sampling.params import SamplingParams
    R, ctx = args.requests, args.context
    page = ModelRunner.default_page_size
    runner = ModelRunner.from_random(cfg, seed=0, dtype="bfloat16", device="cuda:0",
                                     num_pages=R * (-(-(2048 + args.max_tokens + 1) // page)) + 8, max_requests=R,
                                     max_batched_tokens=8192, max_context=ctx, validate=False)
    eng = Engine(runner, SchedulerConfig(max_concurrent_seqs=R, max_batched_tokens=8192, prefill_chunk_tokens=2048,
                                         max_context=ctx))
    gen = torch.Generator().manual_seed(7)
    lens = torch.randint(128, 2049, (R,), generator=gen).tolist()

    def one_round(tag):
        for i, n in enumerate(lens):
            eng.admit((tag, i), torch.randint(0, cfg["vocab_size"], (n,), generator=gen).tolist(),
                      SamplingParams(temperature=0.0, max_tokens=args.max_tokens, ignore_eos=True))
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        done = eng.run()
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        assert len(done) == R and all(len(f.tokens) == args.max_tokens for f in done), eng.last_error
        return dt

    one_round("warm")           # compiles nothing new afterwards: graphs of every bucket are captured
    steps0 = eng.stats.steps
    dt = one_round("timed")
    runner.check_status()
    out_toks, in_toks = R * args.max_tokens, sum(lens)
    print(json.dumps({"only": "serve", "model": "LFM2-%s sizes" % args.sizes.upper(), "requests": R,
                      "prompt_tokens": in_toks, "generated_tokens": out_toks, "seconds": round(dt, 4),
                      "generated_tokens_per_s": round(out_toks / dt, 1),
                      "all_tokens_per_s": round((in_toks + out_toks) / dt, 1),
                      "steps": eng.stats.steps - steps0, "preemptions": eng.stats.preemptions,
                      "steps_ahead": eng.stats.ahead_steps}), flush=True)
    return 0


def measure_prefill(runner, ops, mm_params, pk, peak_tflops, gen, vocab, dev, warm=3, iters=5, families=True):
    """One 2,048-token prompt in one step, L2 flushed before each timed run; then, once more, with
    CUDA events around every kernel call of the step: where the time goes, family by family."""
    import torch
    from vapi_b200.engine.step import StepEntry
    T = 2048
    flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device=dev)

    def one(tag):
        rc = runner.cache.open(("prefill", tag))
        toks = torch.randint(0, vocab, (T,), generator=gen).tolist()
        assert runner.cache.reserve(rc, T)
        flush.zero_()                                   # larger than L2: nothing of the last run stays cached
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        runner.step([StepEntry(rc, toks, [T - 1])])
        e1.record()
        torch.cuda.synchronize()
        runner.cache.close(rc)
        return e0.elapsed_time(e1)

    times = [one(it) for it in range(warm + iters)][warm:]
    pre_ms = sorted(times)[len(times) // 2]
    n_attn_sites = [s for g in runner.cache.paged for s in g.sites]
    head_params = runner.plan.head.weight.numel()
    attn_flops = 0.0
    for g in runner.cache.paged:
        # per attention call site: QK^T and PV over the causal half, 2 flops a multiply-add
        mixers = [runner.plan.layers[runner.plan.order[s].layer].mixer for s in g.sites]
        attn_flops += sum(4.0 * m.nh * m.d * (T * (T + 1) / 2) for m in mixers)
    flops = 2.0 * (mm_params - head_params) * T + 2.0 * head_params * 1 + attn_flops
    prefill = {"value": round(T / (pre_ms / 1e3), 1), "tokens": T, "ms": round(pre_ms, 3),
               "frac": round(flops / (pre_ms / 1e3) / (peak_tflops * 1e12), 4),
               "tflops": round(flops / (pre_ms / 1e3) / 1e12, 1), "peak_tflops": peak_tflops}
    print(f"[bench] prefill: {prefill}", file=sys.stderr, flush=True)
    fam_out = None
    if families:
        with OpLog(ops, runner.plan, events=True) as log:
            total = one("families")
        fam = {}
        for c in log.calls:
            f = fam.setdefault(family_of(c), {"ms": 0.0, "flops": 0.0, "bytes": 0, "calls": 0})
            f["ms"] += c["events"][0].elapsed_time(c["events"][1])
            f["calls"] += 1
            if c["op"] in PRODUCTS and c["weight_shape"]:
                f["flops"] += 2.0 * c["rows"] * c["weight_shape"][0] * c["weight_shape"][1]
            elif c["op"] in ("paged_attention", "decode_attention_fused"):
                f["flops"] += attn_flops / max(1, len(n_attn_sites))
            else:
                f["bytes"] += c["moved_bytes"]
        fam_out = {"ms_with_events": round(total, 3)}
        for name, f in sorted(fam.items(), key=lambda kv: -kv[1]["ms"]):
            row = {"ms": round(f["ms"], 3), "calls": f["calls"]}
            if f["flops"]:
                tf = f["flops"] / (f["ms"] / 1e3) / 1e12
                row.update(tflops=round(tf, 1), frac_peak=round(tf / peak_tflops, 3))
            else:
                gb = f["bytes"] / (f["ms"] / 1e3) / 1e9
                row.update(GBps=round(gb, 0), frac_hbm=round(gb / pk["hbm_gbs"], 3))
            fam_out[name] = row
    return prefill, fam_out


def vukavik_sizes(name):
    """Vukavik layers at the widths of LFM2-<name>: attention with the same heads as the LFM2 stack
    (keys and values of 64, chunks of 8,192, YaRN-scaled rotation), the gated delta rule with heads of
    128 x 128 across the width, Mamba-2 with twice the width inside (heads of 64, state 128), a dense
    feed-forward of the LFM2 stack's width behind every mixer; eight layers."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    mlp = {"kind": "dense", "ff": ff}
    att = {"type": "attention", "mlp": mlp, "mixer": {
        "heads": lf["num_attention_heads"], "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64, "scale": 0.125,
        "mask": {"size": 8192}, "rot": {"base": 1000000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    dl = {"type": "delta", "mlp": mlp, "mixer": {"heads": W // 128, "kv_heads": W // 128, "dim": 128, "vdim": 128, "conv": 4}}
    mb = {"type": "mamba2", "mlp": mlp, "mixer": {"heads": 2 * W // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}}
    vk = {"architecture": "Vukavik", "vocab": lf["vocab_size"], "width": W, "residual_mult": 0.5, "logit_scale": 1.0,
          "norm": {"eps": 1e-5}, "layers": [dl, mb, dl, att, dl, mb, dl, att]}
    lf = dict(lf, num_hidden_layers=8, layer_types=["conv", "conv", "conv", "full_attention"] * 2)
    return vk, lf


def rapolix_sizes(name):
    """Rapolix layers at the widths of LFM2-<name>: two residual streams; in every layer attention with the same
    heads as the LFM2 stack (keys and values of 64) over a window of 1,024 that keeps the first four tokens, beside
    a recurrent block as wide as the model in parts of 256 with a convolution of four taps; feed-forwards
    alternate between a dense one of the LFM2 stack's width and a mixture of 30 experts and 2 identity experts
    (a quarter of that width each, four of them a token, from two of four groups) with a shared expert; eight layers."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    mixer = {"left": {"heads": lf["num_attention_heads"], "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64,
                      "scale": 0.125, "mask": {"size": 1024, "keep_first": 4}},
             "right": {"width": W, "blocks": W // 256, "conv": 4}}
    dense = {"type": "parallel", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}}
    sparse = {"type": "parallel", "mixer": mixer, "mlp": {
        "kind": "moe", "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4},
        "router": {"experts": 30, "identity": 2, "top": 4, "groups": {"count": 4, "keep": 2}}}}
    rp = {"architecture": "Rapolix", "vocab": lf["vocab_size"], "width": W, "streams": 2, "logit_softcap": 50.0,
          "norm": {"eps": 1e-5}, "layers": [dense, sparse] * 4}
    lf = dict(lf, num_hidden_layers=8, layer_types=["conv", "conv", "conv", "full_attention"] * 2)
    return rp, lf


def demazen_sizes(name):
    """Demazen layers at the widths of LFM2-<name>: the matrix memory with heads of 128 x 256 (keys half as wide as
    the model in all, values as wide as it); attention with the same heads as the LFM2 stack (keys and values of 64, q
    and k normed over their whole projections, no rotation) over a window of 1,024 beside gated linear attention
    with four heads of 128 x 256 and a decay through a pair of rank 16; feed-forwards alternate between a dense one of
    the LFM2 stack's width and a mixture of 32 experts (a quarter of that width each, four of them a token); learned
    positions; eight layers, the last two running the weights of the two before them.  Beside it Vukavik (the
    matrix-state recurrences of the package: gated delta rule, Mamba-2) and Rapolix (window attention beside a
    recurrence, experts) at the same widths."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    dense = {"kind": "dense", "ff": ff}
    sparse = {"kind": "moe", "expert": {"ff": ff // 4}, "router": {"experts": 32, "top": 4}}
    memory = {"heads": W // 256, "dim": 128, "vdim": 256, "gate_cap": 15.0}
    par = {"left": {"heads": lf["num_attention_heads"], "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64,
                    "scale": 0.125, "mask": {"size": 1024}},
           "right": {"heads": 4, "dim": 128, "vdim": 256, "tau": 16.0, "rank": 16}}
    layers = [{"type": "mlstm", "mixer": memory, "mlp": dense}, {"type": "parallel", "mixer": par, "mlp": sparse},
              {"type": "mlstm", "mixer": memory, "mlp": sparse}, {"type": "parallel", "mixer": par, "mlp": dense}] * 2
    layers[6], layers[7] = dict(layers[6], weights_of=4), dict(layers[7], weights_of=5)
    dz = {"architecture": "Demazen", "vocab": lf["vocab_size"], "width": W, "max_positions": 8192, "logit_softcap": 30.0,
          "norm": {"eps": 1e-5}, "layers": layers}
    return dz, vukavik_sizes(name)[0], rapolix_sizes(name)[0]


def nelosun_sizes(name):
    """Nelosun layers at the widths of LFM2-<name>: attention with the same heads as the LFM2 stack (keys and values of
    64, a sink, a gate per head, biases, a query temperature that steps every 1,024 positions); latent attention with
    as many heads of 64 + 32 (values of 64) over a cached row of 256 + 32 and a query latent of three eighths of the
    width; a recurrent block as wide as the model in parts of 256 with a convolution of four taps; behind every mixer
    a mixture of 16 gated experts with clamped activations (a quarter of the LFM2 stack's feed-forward width each, four
    of them a token, chosen by a table over the token ids); eight layers in one pass of the loop, so that the input
    product runs once.  Beside it Rapolix (general attention beside the same recurrent block, squared-ReLU experts
    behind a router) and Demazen (gated experts behind a router) at the same widths."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    heads = lf["num_attention_heads"]
    mlp = {"kind": "moe", "expert": {"ff": ff // 4, "limit": 7.0}, "router": {"experts": 16, "top": 4}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64,
                                                      "scale": 0.125, "q_temp": {"coef": 0.1, "every": 1024}}}
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256,
                                                             "q_rank": 3 * W // 8, "scale": 0.1, "rot": {"base": 10000.0, "dims": 32}}}
    rec = {"type": "rglru", "mlp": mlp, "mixer": {"width": W, "blocks": W // 256, "conv": 4}}
    ne = {"architecture": "Nelosun", "vocab": lf["vocab_size"], "width": W, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
          "loop": {"start": 0, "stop": 8, "times": 1}, "layers": [lat, att, rec, att] * 2}
    return ne, rapolix_sizes(name)[0], demazen_sizes(name)[0]


def givavik_sizes(name):
    """Givavik layers at the widths of LFM2-<name>: latent attention with as many heads as the LFM2 stack, of 64 + 32
    (values of 64), over a cached row of 256 + 32, every second such layer reading the latents of the one before it;
    attention with the same heads as the LFM2 stack (keys and values of 64, sigmoid weights, a cap of 40) beside Mamba-2
    with twice the width inside (heads of 64, state 128); a dense feed-forward of the LFM2 stack's width with xIELU beside
    every mixer; a bigram table; eight layers.  Beside it Nelosun (latent attention, attention on the same kernels with a
    softmax, the same arrangement of a layer) and Vukavik (Mamba-2, attention, dense feed-forwards) at the same widths."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    heads = lf["num_attention_heads"]
    mlp = {"kind": "dense", "ff": ff}

    def lat(source=None):
        m = {"heads": heads, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "scale": 0.1, "rot": {"base": 10000.0, "dims": 32}}
        return {"type": "latent_attention", "mlp": mlp, "mixer": m if source is None else dict(m, kv_from=source)}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64, "scale": 0.125, "softcap": 40.0,
                 "rot": {"base": 10000.0, "dims": 64}},
        "right": {"heads": 2 * W // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1},
        "left_scale": 0.8, "right_scale": 1.25}}
    gv = {"architecture": "Givavik", "vocab": lf["vocab_size"], "width": W, "norm": {"eps": 1e-5},
          "embedding": {"scale": 1.0, "bigram": {"buckets": 16381, "mul_prev": 31337, "mul_cur": 911}},
          "layers": [lat(), par, lat(0), par, lat(), par, lat(4), par]}
    return gv, nelosun_sizes(name)[0], vukavik_sizes(name)[0]


def zokelorn_sizes(name):
    """Zokelorn layers at the widths of LFM2-<name>: lightning attention with heads of 128 x 128 across the width; retention
    with heads of 128 x 256 (keys half as wide as the model in all, values as wide as it); attention with the same heads as
    the LFM2 stack (keys and values of 64, chunks of 8,192, a gate per head, stretched frequencies); feed-forwards alternate
    between a dense one of the LFM2 stack's width and a mixture of 32 experts (a quarter of that width each, four of them a
    token, from two of four groups) with a gated shared expert of that quarter; eight layers in one pass of the loop.  Beside
    it Demazen (matrix-state recurrences with the same states, gated experts behind a router, dense feed-forwards) and
    Nelosun (attention on the same kernels, the same arrangement of a layer, gated experts) at the same widths."""
    from vapi_b200.models.lfm2 import Lfm2Config
    lf = lfm2_sizes(name)
    W, ff = lf["hidden_size"], Lfm2Config.effective_ff_dim(lf)
    dense = {"kind": "dense", "ff": ff}
    sparse = {"kind": "moe", "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4},
              "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}}}
    lin = {"heads": W // 128, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-1.0 - 8.0 * h * 128 / W) for h in range(W // 128)]}
    ret = {"heads": W // 256, "dim": 128, "vdim": 256, "decay": [1.0 - 2.0 ** (-5.0 - h) for h in range(W // 256)]}
    att = {"heads": lf["num_attention_heads"], "kv_heads": lf["num_key_value_heads"], "dim": 64, "vdim": 64, "scale": 0.125,
           "mask": {"size": 8192}, "rot": {"base": 500000.0, "dims": 64,
                                           "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    layers = [{"type": "lightning", "mixer": lin, "mlp": dense}, {"type": "retention", "mixer": ret, "mlp": sparse},
              {"type": "lightning", "mixer": lin, "mlp": sparse}, {"type": "attention", "mixer": att, "mlp": dense}] * 2
    zk = {"architecture": "Zokelorn", "vocab": lf["vocab_size"], "width": W, "norm": {"eps": 1e-5},
          "loop": {"start": 0, "stop": 8, "times": 1}, "layers": layers}
    return zk, demazen_sizes(name)[0], nelosun_sizes(name)[0]


def mixers(args):
    """``--only mixers``: prefill and decode of eight layers of ``--design`` beside LFM2 layers (Vukavik, Rapolix; Demazen
    stands beside Vukavik and Rapolix, whose kernels are the nearest to its own, Nelosun beside Rapolix and Demazen, Givavik
    beside Nelosun and Vukavik, Zokelorn beside Demazen and Nelosun)
    of equal width (random weights), and where each model's time goes, kernel family by kernel family."""
    import torch
    from vapi_b200 import ops
    from vapi_b200.engine.runner import ModelRunner
    from vapi_b200.engine.step import StepEntry
    pk = peaks()
    dev = torch.device("cuda:0")
    torch.cuda.set_device(dev)
    T, B, ctx_len, page = 2048, args.batch, min(args.context, 4096), args.page_size or ModelRunner.default_page_size
    gen = torch.Generator().manual_seed(1)
    flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device=dev)
    out = {"only": "mixers", "sizes": args.sizes, "dtype": "bfloat16", "prefill_tokens": T, "decode_batch": B,
           "decode_context": ctx_len, "peaks": pk, "models": {}}
    out["design"] = args.design
    if args.design == "demazen":
        dz, vk, rp = demazen_sizes(args.sizes)
        models = (("demazen", dz), ("vukavik", vk), ("rapolix", rp))
    elif args.design == "nelosun":
        ne, rp, dz = nelosun_sizes(args.sizes)
        models = (("nelosun", ne), ("rapolix", rp), ("demazen", dz))
    elif args.design == "givavik":
        gv, ne, vk = givavik_sizes(args.sizes)
        models = (("givavik", gv), ("nelosun", ne), ("vukavik", vk))
    elif args.design == "zokelorn":
        zk, dz, ne = zokelorn_sizes(args.sizes)
        models = (("zokelorn", zk), ("demazen", dz), ("nelosun", ne))
    else:
        vk, lf = rapolix_sizes(args.sizes) if args.design == "rapolix" else vukavik_sizes(args.sizes)
        models = ((args.design, vk), ("lfm2", lf))
    for name, cfg in models:
        vocab = cfg.get("vocab") or cfg["vocab_size"]
        n_pages = (B + 1) * (-(-(ctx_len + 64) // page)) + 8
        runner = ModelRunner.from_random(cfg, seed=0, dtype="bfloat16", device="cuda:0", num_pages=n_pages, page_size=page,
                                         max_requests=max(B, 8), max_batched_tokens=8192, max_context=ctx_len + 64,
                                         watermark=0.0, validate=False)
        wbytes, mm_params = model_numbers(runner)

        def prefill(tag, log=None):
            rc = runner.cache.open(("p", tag))
            toks = torch.randint(0, vocab, (T,), generator=gen).tolist()
            assert runner.cache.reserve(rc, T)
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            e0.record()
            runner.step([StepEntry(rc, toks, [T - 1])])
            e1.record()
            torch.cuda.synchronize()
            runner.cache.close(rc)
            return e0.elapsed_time(e1)

        times = [prefill(i) for i in range(3 + 5)][3:]
        pre_ms = sorted(times)[len(times) // 2]
        with OpLog(ops, runner.plan, events=True) as log:
            prefill("families")
        torch.cuda.synchronize()
        fam = {}
        for c in log.calls:
            f = fam.setdefault(family_of(c), {"ms": 0.0, "calls": 0, "flops": 0.0, "bytes": 0})
            f["ms"] += c["events"][0].elapsed_time(c["events"][1])
            f["calls"] += 1
            if c["op"] in PRODUCTS and c["weight_shape"]:
                f["flops"] += 2.0 * c["rows"] * c["weight_shape"][0] * c["weight_shape"][1]
            else:
                f["bytes"] += c["moved_bytes"]
        # arithmetic of the mixers' own kernels for one prompt of T tokens, per call
        mix_flops = {}
        for blk in runner.plan.layers:
            ffn = getattr(blk, "ffn", None)
            if type(ffn).__name__ == "SparseMoE":
                # (as if every choice were an expert; a gated expert has three matrices)
                mix_flops["moe_experts"] = 2.0 * (3 if ffn.gated else 2) * ffn.top * ffn.ff * ffn.hidden * T
                mix_flops["moe_route"] = 2.0 * (ffn.E + ffn.I) * ffn.hidden * T
        for blk in runner.plan.layers:
          for m in blk.mixer.members():
            kind = type(m).__name__
            if kind == "GQAttention" and getattr(m, "window", 0) > 0 and not getattr(m, "chunk", 0):
                pairs = sum(min(t + 1, m.window + min(m.keep_first, max(0, t + 1 - m.window))) for t in range(T))
                mix_flops["masked_attention" if m.general else "paged_attention"] = 2.0 * m.nh * (m.d + m.dv) * pairs
            elif kind == "RGLRUMixer":
                mix_flops["rglru"] = 2.0 * 2 * m.C * (m.C // m.B) * T                        # the two gates' products
            elif kind == "LatentAttention":
                # a score over the whole cached row, a weighted sum over its latent
                mix_flops["latent_attention"] = 2.0 * m.H * (2 * m.R + m.r) * T * (T + 1) / 2
                mix_flops["head_products"] = 2.0 * m.H * m.R * (m.d + m.dv) * T / 2         # two calls a layer: their mean
            elif kind == "GQAttention":
                span = min(T, m.chunk) if getattr(m, "chunk", 0) else T
                pairs = (T // span) * span * (span + 1) / 2 + (T % span) * (T % span + 1) / 2
                mix_flops["masked_attention" if getattr(m, "general", False) else "paged_attention"] = 2.0 * m.nh * (m.d + getattr(m, "dv", m.d)) * pairs
            elif kind == "GatedDeltaMixer":
                mix_flops["gated_delta"] = 2.0 * 4 * m.nh * m.dk * m.dv * T      # decay, S^T k, the rank-one write, S^T q
            elif kind == "Mamba2Mixer":
                mix_flops["state_space"] = 2.0 * 3 * m.nh * m.N * m.p * T        # decay, the rank-one write, S^T C
            elif kind == "MatrixMemoryMixer":
                mix_flops["matrix_memory"] = 2.0 * 3 * m.nh * m.dk * m.dv * T    # decay, the rank-one write, S^T q
            elif kind == "FixedDecayMixer":
                # (per call, of the token-by-token form; layers of two kinds: their mean)
                mix_flops.setdefault("fixed_decay_each", []).append(2.0 * 3 * m.nh * m.dk * m.dv * T)
                mix_flops["fixed_decay_memory"] = sum(mix_flops["fixed_decay_each"]) / len(mix_flops["fixed_decay_each"])
            elif kind == "GatedLinearAttentionMixer":
                mix_flops["gated_linear_attention"] = 2.0 * 3 * m.nh * m.dk * m.dv * T
        rows = {}
        for k, f in sorted(fam.items(), key=lambda kv: -kv[1]["ms"]):
            row = {"ms": round(f["ms"], 3), "calls": f["calls"]}
            if f["flops"]:
                tf = f["flops"] / (f["ms"] / 1e3) / 1e12
                row.update(tflops=round(tf, 1), frac_bf16_peak=round(tf / pk["bf16_tflops"], 3))
            elif k in mix_flops:
                tf = mix_flops[k] * f["calls"] / (f["ms"] / 1e3) / 1e12
                row.update(tflops=round(tf, 2))
                if "attention" in k:
                    row.update(frac_bf16_peak=round(tf / pk["bf16_tflops"], 4))
            if not f["flops"] and f["bytes"]:
                gb = f["bytes"] / (f["ms"] / 1e3) / 1e9
                row.update(GBps=round(gb, 0), frac_hbm=round(gb / pk["hbm_gbs"], 3))
            rows[k] = row
        # decode: B requests at ctx_len, captured steps
        rcs = []
        start = ctx_len - args.steps - 1
        for i in range(B):
            rc = runner.cache.open(("d", i))
            toks = torch.randint(0, vocab, (start,), generator=gen).tolist()
            pos = 0
            while pos < start:
                q = min(2048, start - pos)
                assert runner.cache.reserve(rc, pos + q)
                runner.step([StepEntry(rc, toks[pos:pos + q], [])])
                pos += q
            rcs.append(rc)

        def decode(count):
            toks = torch.randint(0, vocab, (count, B), generator=gen).tolist()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            before = ops.launch_count
            e0.record()
            for s_ in range(count):
                entries = []
                for j, rc in enumerate(rcs):
                    assert runner.cache.reserve(rc, rc.num_tokens + 1)
                    entries.append(StepEntry(rc, [toks[s_][j]], [0]))
                logits = runner.step_decode_graph(entries)
                if logits is None:
                    logits = runner.step(entries)
                ops.sample_rows(logits)
            e1.record()
            torch.cuda.synchronize()
            return e0.elapsed_time(e1), ops.launch_count - before

        regions = []
        for it in range(2 + 5):
            ms, launches = decode(args.steps)
            for rc in rcs:
                runner.cache.commit(rc, start)
            if it >= 2:
                regions.append(ms)
        dec_ms = sorted(regions)[len(regions) // 2] / args.steps
        kv_bytes = B * ctx_len * runner.cache.bytes_per_token() + B * runner.cache.state_bytes_per_request()
        for rc in rcs:
            runner.cache.close(rc)
        out["models"][name] = {
            "weights_GB": round(wbytes / 1e9, 3),
            "prefill": {"ms": round(pre_ms, 3), "tokens_per_s": round(T / (pre_ms / 1e3), 0),
                        "matrix_tflops": round(2.0 * mm_params * T / (pre_ms / 1e3) / 1e12, 1)},
            "decode": {"ms_per_step": round(dec_ms, 4), "tokens_per_s": round(B / (dec_ms / 1e3), 0),
                       "launches_per_step": launches // args.steps,
                       "frac_hbm": round((wbytes + kv_bytes) / (dec_ms / 1e3) / 1e9 / pk["hbm_gbs"], 3)},
            "prefill_kernels": rows}
        print(f"[bench] {name}: prefill {pre_ms:.3f} ms, decode {dec_ms:.4f} ms/step", file=sys.stderr, flush=True)
        del runner
        torch.cuda.empty_cache()
    print(json.dumps(out), flush=True)
    return 0


def reference_arm():
    """The reference is a Rust workspace (Cargo, candle); it has no Python package to
    install and no Rust toolchain exists here, so its arm cannot run."""
    print(json.dumps({"impl": "reference",
                      "unavailable": "Heyo-Computer/vapi is a Rust/Cargo workspace with no Python packaging; "
                                     "pip cannot install it offline and there is no cargo/rustc in the image"}),
          flush=True)
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=512)
    ap.add_argument("--warmup", type=int, default=32)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration has (0 = all)")
    ap.add_argument("--impl", default="vapi_b200", choices=["vapi_b200", "reference"])
    ap.add_argument("--only", default="all", choices=["all", "decode", "prefill", "serve", "trace", "mixers"],
                    help="run just the headline decode point, just the prefill, (serve) continuous "
                         "batching of --requests requests with random prompt lengths through the engine loop, or "
                         "(trace) a few decode steps of a measuring build whose kernels stamp the device clock, "
                         "and print what one step's kernels did inside the captured graph, or (mixers) prefill and "
                         "decode of eight Vukavik layers beside eight LFM2 layers of equal width, kernel family by kernel family")
    ap.add_argument("--sizes", default="1.2b", choices=["1.2b", "700m", "2.6b"], help="layer sizes of LFM2-<sizes>")
    ap.add_argument("--design", default="vukavik", choices=["vukavik", "rapolix", "demazen", "nelosun", "givavik", "zokelorn"],
                    help="with --only mixers: the architecture whose layers stand beside LFM2's (demazen: beside Vukavik's and "
                         "Rapolix's; nelosun: beside Rapolix's and Demazen's; givavik: beside Nelosun's and Vukavik's; "
                         "zokelorn: beside Demazen's and Nelosun's)")
    ap.add_argument("--page-size", type=int, default=0, help="tokens per cache page (0: the engine's default)")
    ap.add_argument("--dtype", default="bfloat16", help="bfloat16 (serving) or float32 (the true 32-bit path)")
    ap.add_argument("--no-fp32", action="store_true", help="leave the float32 points out of the default run")
    ap.add_argument("--no-kernels", action="store_true", help="leave the decode step's kernel table (a second process) out")
    ap.add_argument("--rows-json", action="store_true", help="with --only trace: one JSON line of named kernels")
    ap.add_argument("--requests", type=int, default=64)
    ap.add_argument("--max-tokens", type=int, default=128)
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    if args.gpus != 1:
        print("bench.py: this engine runs on one GPU; --gpus %d is not supported" % args.gpus, flush=True)
        return 2
    if args.warmup < 3:
        args.warmup = 3
    return run(args)


if __name__ == "__main__":
    sys.exit(main())
