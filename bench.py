"""Decode and prefill throughput of the Llama-3-8B shape on one B200, random weights, bfloat16.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference] [--layers L] [--model NAME]
                    [--dtype bf16|fp32] [--points default|main|long]

Prints ONE JSON line.  ``value``: decoded tokens a second at batch 8 (prompt lengths uniform in
[128, 2048]); after W warm-up steps, ``regions`` (5) regions of K decode steps each are timed on the device
with CUDA events and the median region counts; a step is one decode step, the next token chosen greedily on
the device.  ``e2e``: the same through the Python entry point ``generate`` with host token lists in and out (a
pinned host-to-device copy of every step's tokens and a device-to-host read of every step's result inside the
timed region), again the median of 5 regions of K steps.  ``prefill``: one prompt of 2,048 tokens.
``roofline``: the bytes a decode step has to read (every weight it uses once, and the cache of the live
requests) over its time, against the measured copy bandwidth.  ``points``: tokens a second of decode at batch
1, 16, 32, 64 and 128, of a batch of 64 of which one sequence ends every third step (down to 16; by the clock, host
tokens in, the live set changing under the captured graphs), of decode at batch 8 with 7,000 to 8,000 cached tokens a request, of prefills of 512 and 8,192
tokens, and of the benchmark's further configurations (decode at batch 8 and a prefill of 2,048 tokens for the
Llama-2-7B and Llama-2-13B shapes, decode at batch 8 in float32); ``points_frac``: each point's fraction of its
roofline (copy bandwidth for decode, the dtype's arithmetic peak for prefill).  Weights (15 GB a step) are
larger than L2, so no flush is needed between steps.

``--dtype fp32`` measures the true 32-bit path (FFMA products, float32 cache) in the same line format.
``--points main`` leaves the further configurations out; ``--points long`` adds decode at batch 64 with
7,000 to 8,000 cached tokens a request (a prefill of half a million tokens comes before it).
``--only decode_b<N>`` or ``--only prefill`` prints that part alone (for profilers); ``--only gemm_rows``,
``attention_prefill`` and ``attention_decode`` time single kernels at the model's layer sizes over a range of rows,
tokens or contexts, one JSON line a size.  The default warm-up of 24 steps covers the 80 ms or so that the GPU's
clocks take to come back up after the prefill's power-capped run.

``--model llama-2-7b`` or ``llama-2-13b`` measures the benchmark's further shapes (32 and 40 kv heads: eight and
ten times the keys and values a token) with their own prompt lengths instead of the default.
``--impl reference`` runs the unmodified reference (baseline/_ref) through its own get_model/generate.
For more than one GPU the program says that it has no such path and exits with 2.
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

# The benchmark's shapes (the default is the first) with their registry variants and prompt lengths.
MODELS = {
    "llama-3-8b": dict(name="llama-3-8b", variant="3-8b", label="Llama-3-8B", nlayers=32, emb_dim=4096, nheads=32, kvheads=8,
                       head_dim=128, ffn_hidden=14336, vocab=128256, context=8192, prompts=(128, 2048)),
    "llama-2-7b": dict(name="llama-2-7b", variant="7b", label="Llama-2-7B", nlayers=32, emb_dim=4096, nheads=32, kvheads=32,
                       head_dim=128, ffn_hidden=11008, vocab=32000, context=4096, prompts=(64, 2048)),
    "llama-2-13b": dict(name="llama-2-13b", variant="13b", label="Llama-2-13B", nlayers=40, emb_dim=5120, nheads=40,
                        kvheads=40, head_dim=128, ffn_hidden=13824, vocab=32000, context=4096, prompts=(1024, 1024)),
}
MODEL = MODELS["llama-3-8b"]
PROMPT_MIN, PROMPT_MAX, PREFILL_TOKENS, BATCH = 128, 2048, 2048, 8


def choose_model(name):
    global MODEL, PROMPT_MIN, PROMPT_MAX
    MODEL = MODELS[name]
    PROMPT_MIN, PROMPT_MAX = MODEL["prompts"]


# float32 on the CUDA cores: 148 multiprocessors x 128 lanes x 2 flops x 1.965 GHz (nominal; nobody measured it here)
FP32_TFLOPS_NOMINAL = 148 * 128 * 2 * 1.965e9 / 1e12
REGIONS = 5  # timed regions of --steps steps each; the median counts


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        with open(path) as f:
            p = json.load(f)
        return dict(hbm_gbs=p["hbm_gbs"], bf16_tflops=p["bf16_tflops"], source="measured")
    return dict(hbm_gbs=6650.0, bf16_tflops=1590.0, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([x.strip() for x in line.split(",")])

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        sm = [float(r[0]) for r in self.rows if len(r) >= 6 and r[0].replace(".", "").isdigit()]
        mx = [float(r[1]) for r in self.rows if len(r) >= 6 and r[1].replace(".", "").isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) >= 6 and r[2 + i].lower() == "active" for r in self.rows)]
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(sm)}


def prompt_lengths(batch, seed=0):
    import numpy as np

    rng = np.random.default_rng(seed + batch)
    return [int(x) for x in rng.integers(PROMPT_MIN, PROMPT_MAX + 1, size=batch)]


def random_prompts(lengths, vocab, seed=0):
    import numpy as np

    rng = np.random.default_rng(1000 + seed)
    return [[int(t) for t in rng.integers(0, vocab, size=n)] for n in lengths]


def decode_bytes(nlayers, batch_context_tokens, m=None, itemsize=2):
    """Bytes one decode step has to read: every weight it uses once, and the cache of the live requests."""
    m = m or MODEL
    d, hd, h, kv, f, v = m["emb_dim"], m["head_dim"], m["nheads"], m["kvheads"], m["ffn_hidden"], m["vocab"]
    per_layer = ((h + 2 * kv) * hd * d + h * hd * d + 2 * f * d + f * d + 2 * d) * itemsize
    weights = nlayers * per_layer + d * itemsize + v * d * itemsize
    cache = batch_context_tokens * nlayers * 2 * kv * hd * itemsize
    return weights + cache


def prefill_flops(nlayers, tokens, m=None):
    m = m or MODEL
    d, hd, h, kv, f, v = m["emb_dim"], m["head_dim"], m["nheads"], m["kvheads"], m["ffn_hidden"], m["vocab"]
    gemm = 2 * tokens * ((h + 2 * kv) * hd * d + h * hd * d + 3 * f * d) * nlayers
    attention = 2 * tokens * tokens * hd * h * nlayers  # causal half of 4 T^2 hd per head
    return gemm + attention + 2 * v * d


# --------------------------------------------------------------------------------------------------
# this library
# --------------------------------------------------------------------------------------------------
def run_kernels(args):
    """--only gemm_rows / attention_prefill / attention_decode: single kernels at the model's layer sizes over a
    range of rows, tokens or contexts, timed alone with CUDA events (L2 flushed before every launch), the products
    beside the library's.  One JSON line a size."""
    import torch

    from fms_b200.cache import Cache, KVRequest
    from fms_b200.engine.batch import Batch
    from fms_b200.kernels import ops

    m = MODEL
    d, hd, h, kv, f = m["emb_dim"], m["head_dim"], m["nheads"], m["kvheads"], m["ffn_hidden"]
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def timed(fn, repeats=10):
        for _ in range(3):
            fn()
        us = []
        for _ in range(repeats):
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            us.append(a.elapsed_time(b) * 1e3)
        return round(statistics.median(us), 1)

    bf16 = torch.bfloat16
    if args.only == "gemm_rows":
        # every own kernel that takes the size, called directly (whatever the step would choose), beside the library
        shapes = {"qkv": ((h + 2 * kv) * hd, d), "dense": (d, h * hd), "down": (d, f)}
        ws = {k: (torch.randn(n, kk, device="cuda") * 0.02).to(bf16) for k, (n, kk) in shapes.items()}
        wg = (torch.randn(2 * f, d, device="cuda") * 0.02).to(bf16)
        ops.USE_MID_GEMM, ops.MID_OPS, ops.MID_ROWS = True, ["linear", "glu", "qkv"], 256
        for rows in (1, 8, 16, 64, 256, 512, 1024, 2048, 4096):
            xs = {d: torch.randn(rows, d, device="cuda").to(bf16), f: torch.randn(rows, f, device="cuda").to(bf16)}
            line = {"only": "gemm_rows", "rows": rows, "us": "weight-streaming (<= 8 rows: mma.sync; 9-256: tcgen05, "
                    "weights on the rows), tcgen05 with the tokens on the rows (>= 128), library"}
            small, large = rows <= 256, rows >= 128
            for name, (n, kk) in shapes.items():
                line[name] = [timed(lambda: ops.linear(xs[kk], ws[name])) if small else None,
                              timed(lambda: ops.linear_tensor_core(xs[kk], ws[name])) if large else None,
                              timed(lambda: torch.nn.functional.linear(xs[kk], ws[name]))]
            line["glu"] = [timed(lambda: ops.gated_linear(xs[d], wg, None, 0)) if small else None,
                           timed(lambda: ops.gated_linear_tensor_core(xs[d], wg, None, 0)) if large else None,
                           timed(lambda: ops.gated_activation(torch.nn.functional.linear(xs[d], wg), 0))]
            print(json.dumps(line), flush=True)
    else:
        cases = [(1, n) for n in (512, 1024, 2048, 4096, 8192)] if args.only == "attention_prefill" else \
            [(b, n) for b, n in ((1, 1024), (1, 8192), (8, 1155), (8, 8192), (64, 1155), (64, 4096))]
        for b, n in cases:
            decode = args.only == "attention_decode"
            cache = Cache([KVRequest(kv, hd, 0)], max_tokens=b * (n + 128), max_positions=n + 128, dtype=bf16, device="cuda")
            slots = cache.begin(b)
            if decode:
                cache.prepare(slots, [n] * b)
                cache.commit(slots, [n] * b)
            new = 1 if decode else n
            cache.prepare(slots, [new] * b)
            view = cache.layer_view(0)
            view.keys.normal_()
            view.values.normal_()
            batch = Batch.from_lists(slots, [n if decode else 0] * b, [[0] * new] * b, [[]] * b, "cuda")
            q = torch.randn(b * new, h * hd, device="cuda").to(bf16)
            us = timed(lambda: ops.attention(q, batch, view, h, kv, hd, hd ** -0.5, 0), repeats=20)
            line = {"only": args.only, "sequences": b, "tokens": n, "us": us}
            if decode:
                line["kv_GBs"] = round(b * n * kv * hd * 2 * 2 / us / 1e3, 1)
            else:
                line["tflops"] = round(4.0 * n * n / 2 * hd * h / us / 1e6, 1)
            print(json.dumps(line), flush=True)
            del cache, view
    ops.check_error_flag("cuda")


class Measured:
    """One model on the device with an engine, and the measurements taken on it."""

    def __init__(self, model_info, dtype, nlayers, room, max_prompt, slots=64, long_requests=0):
        """``room``: decode steps a request goes through; ``long_requests``: how many requests of up to the model's
        whole context the cache has to hold beside ``slots`` requests of ``max_prompt`` tokens."""
        import torch

        from fms_b200.models import get_model

        self.m, self.dtype, self.nlayers = model_info, dtype, nlayers
        self.itemsize = 2 if dtype == "bf16" else 4
        self.model = get_model("llama", model_info["variant"], device_type="cuda", data_type=dtype, seed=0, nlayers=nlayers)
        cfg = self.model.config
        assert (cfg.emb_dim, cfg.nheads, cfg.n_kvheads, cfg.ffn_hidden, cfg.src_vocab_size, cfg.max_expected_seq_len) == (
            model_info["emb_dim"], model_info["nheads"], model_info["kvheads"], model_info["ffn_hidden"], model_info["vocab"],
            model_info["context"])
        self.engine = self.model.new_engine(max_tokens=max(slots * (max_prompt + 2 * room + 128),
                                                           long_requests * model_info["context"]), max_slots=slots)
        self.torch = torch

    def close(self):
        self.engine = self.model = None
        self.torch.cuda.empty_cache()

    def device_decode(self, batch, steps, warmup, lengths=None, regions=REGIONS):
        """(tokens a second, ms a step, mean context, own kernels launched, ms a step of every region): after the
        prompts and ``warmup`` decode steps, ``regions`` regions of ``steps`` decode steps, each between two CUDA events;
        the median region counts."""
        from fms_b200.kernels import ops

        torch, engine = self.torch, self.engine
        lengths = lengths or prompt_lengths(batch)
        prompts = random_prompts(lengths, self.m["vocab"])
        slots = engine.begin(batch)
        try:
            warmup = max(3, warmup)
            horizon = max(lengths) + warmup + regions * steps + 1
            if sum(lengths) > 100_000:  # many long prompts: eight requests a step
                for i in range(0, batch, 8):
                    last = engine.step(slots[i:i + 8], prompts[i:i + 8])
                    logits = last if i == 0 else torch.cat([logits, last])
            else:
                logits = engine.step(slots, prompts)
            tokens = ops.argmax(logits)
            for _ in range(warmup):
                tokens = ops.argmax(engine.decode(slots, tokens_device=tokens, horizon=horizon))
            torch.cuda.synchronize()
            context = sum(engine.length(s) for s in slots) + batch * (regions * steps + 1) / 2.0
            launches0, graphs0 = ops.launches, engine.graph_launches
            events = [torch.cuda.Event(enable_timing=True) for _ in range(regions + 1)]
            events[0].record()
            for r in range(regions):
                for _ in range(steps):
                    tokens = ops.argmax(engine.decode(slots, tokens_device=tokens, horizon=horizon))
                events[r + 1].record()
            torch.cuda.synchronize()
            per_region = [events[r].elapsed_time(events[r + 1]) / steps for r in range(regions)]
            ms = statistics.median(per_region)
            launched = ((ops.launches - launches0) + (engine.graph_launches - graphs0) * engine.kernels_per_graph) // regions
            engine.check()
        finally:
            engine.release(slots)
        return batch / (ms / 1e3), ms, context, launched, per_region

    def ending_decode(self, batch=64, every=3, until=16):
        """Tokens a second of a batch whose sequences end one by one (one every ``every`` steps, down to ``until``):
        host tokens in and out as a generation loop has them, timed by the clock from the first decode step to the
        last, the second of two passes (the first leaves the graphs of the sizes captured, as a running engine has them)."""
        import random as _random
        import time as _time

        torch, engine = self.torch, self.engine
        lengths = prompt_lengths(batch)
        prompts = random_prompts(lengths, self.m["vocab"])
        value = 0.0
        for _ in range(2):
            rng = _random.Random(3)
            slots = engine.begin(batch)
            live = list(slots)
            try:
                engine.step(slots, prompts)
                horizon = max(lengths) + every * batch
                torch.cuda.synchronize()
                start, done, step = _time.perf_counter(), 0, 0
                while len(live) > until:
                    step += 1
                    if step % every == 0:
                        engine.release([live.pop(rng.randrange(len(live)))])
                    engine.decode(live, [1] * len(live), horizon=horizon)
                    done += len(live)
                torch.cuda.synchronize()
                value = done / (_time.perf_counter() - start)
                engine.check()
            finally:
                engine.release(live)
        return value

    def host_decode(self, batch, steps, warmup, regions=REGIONS):
        """The same through generate(): host token lists in, host tokens out, every step."""
        from fms_b200.utils.generation import generate

        torch, engine = self.torch, self.engine
        lengths = prompt_lengths(batch)
        prompts = [torch.tensor(p) for p in random_prompts(lengths, self.m["vocab"])]
        h2d0 = engine.h2d_bytes
        _, times = generate(engine, prompts, max_new_tokens=1 + max(3, warmup) + regions * steps, do_sample=False,
                            timing="per-token")
        timed = times[-regions * steps:]
        per_region = [sum(timed[r * steps:(r + 1) * steps]) for r in range(regions)]
        h2d_decode = 4 * batch  # each decode step copies its tokens from a pinned host array
        assert engine.h2d_bytes - h2d0 >= h2d_decode * regions * steps
        return batch * steps / statistics.median(per_region), h2d_decode, 4 * batch

    def prefill(self, tokens, repeats=5):
        torch, engine = self.torch, self.engine
        prompt = random_prompts([tokens], self.m["vocab"], seed=7)
        ms = []
        for i in range(3 + repeats):  # three warm-up runs, then the timed ones
            (slot,) = engine.begin(1)
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            engine.step([slot], prompt)
            end.record()
            torch.cuda.synchronize()
            engine.release([slot])
            if i >= 3:
                ms.append(start.elapsed_time(end))
        return statistics.median(ms)

    def decode_frac(self, ms_step, context, pk):
        return decode_bytes(self.nlayers, context, self.m, self.itemsize) / (ms_step / 1e3) / 1e9 / pk["hbm_gbs"]

    def prefill_frac(self, ms, tokens, pk):
        peak = pk["bf16_tflops"] if self.dtype == "bf16" else FP32_TFLOPS_NOMINAL
        return prefill_flops(self.nlayers, tokens, self.m) / (ms / 1e3) / (peak * 1e12)


def run_ours(args):
    import numpy as np

    pk = peaks()
    dtype = args.dtype
    nlayers = args.layers or MODEL["nlayers"]
    room = max(3, args.warmup) + REGIONS * args.steps + 8
    long_context = args.points != "main" and not args.only and MODEL["context"] >= 8192
    # 128 slots (for the point at batch 128) where their cache stays well inside the memory: the 8B shape in bfloat16
    # holds 128 KB a token, the shapes with as many kv heads as heads four times that
    token_bytes = 2 * nlayers * MODEL["kvheads"] * MODEL["head_dim"] * (2 if dtype == "bf16" else 4)
    roomy = 128 * (PROMPT_MAX + 2 * room + 128) * token_bytes < 60e9
    slots = max(64, int(args.only.split("_b")[1])) if args.only.startswith("decode_b") else (128 if roomy else 64)
    run = Measured(MODEL, dtype, nlayers, room, PROMPT_MAX, slots=slots,
                   long_requests=(64 if args.points == "long" else 8) if long_context else 0)

    if args.only:  # a short run of one part, for profilers: prints that part's figures only
        if args.only == "prefill":
            print(json.dumps({"only": "prefill", "tokens": args.prefill_tokens,
                              "ms": round(run.prefill(args.prefill_tokens, repeats=args.steps), 3)}))
        else:
            batch = int(args.only.split("_b")[1])
            v, ms, _, _, _ = run.device_decode(batch, args.steps, args.warmup, regions=1)
            e2e, _, _ = run.host_decode(batch, args.steps, args.warmup, regions=1)
            print(json.dumps({"only": args.only, "value": round(v, 1), "ms_per_step": round(ms, 4), "e2e": round(e2e, 1)}))
        return
    sampler = ClockSampler()
    sampler.start()
    value, ms_step, context, launched, per_region = run.device_decode(BATCH, args.steps, args.warmup)
    e2e, h2d, d2h = run.host_decode(BATCH, args.steps, args.warmup)
    sampler.stop()
    points, fracs = {}, {}

    def decode_point(name, r, batch, steps, lengths=None, regions=3):
        v, ms, ctx, _, _ = r.device_decode(batch, steps, args.warmup, lengths, regions)
        points[name], fracs[name] = round(v, 1), round(r.decode_frac(ms, ctx, pk), 4)

    def prefill_point(name, r, tokens, repeats=3):
        ms = r.prefill(tokens, repeats)
        points[name], fracs[name] = round(tokens / (ms / 1e3), 1), round(r.prefill_frac(ms, tokens, pk), 4)

    side = max(32, args.steps // 2)
    for b in (1, 16, 32, 64) + ((128,) if slots >= 128 else ()):
        decode_point(f"decode_b{b}", run, b, side)
    points["decode_b64_ending_one_by_one"] = round(run.ending_decode(), 1)
    pf_ms = run.prefill(PREFILL_TOKENS)
    prefill_point("prefill_512", run, 512)
    if long_context:
        rng = np.random.default_rng(5)
        prefill_point("prefill_8192", run, 8192)
        decode_point("decode_b8_ctx8192", run, 8, side, [int(x) for x in rng.integers(7000, 8000 - 3 * side - 32, size=8)])
        if args.points == "long":
            decode_point("decode_b64_ctx8192", run, 64, side, [int(x) for x in rng.integers(7000, 8000 - 3 * side - 32, size=64)])
    gbs = decode_bytes(nlayers, context, MODEL, run.itemsize) / (ms_step / 1e3) / 1e9
    pf_frac = run.prefill_frac(pf_ms, PREFILL_TOKENS, pk)
    run.close()
    if args.points != "main" and args.model == "llama-3-8b" and not args.layers:
        # the benchmark's further configurations, each on a model of its own: decode at batch 8 and one prefill
        others = [("l2_7b", MODELS["llama-2-7b"], "bf16"), ("l2_13b", MODELS["llama-2-13b"], "bf16")]
        others.append(("fp32", MODELS["llama-3-8b"], "fp32") if dtype == "bf16" else ("bf16", MODELS["llama-3-8b"], "bf16"))
        for tag, info, dt in others:
            lo, hi = info["prompts"]
            rng = np.random.default_rng(8)
            lengths = [int(x) for x in rng.integers(lo, hi + 1, size=BATCH)]
            steps = side if dt == "bf16" else 8
            other = Measured(info, dt, info["nlayers"], max(3, args.warmup) + 3 * steps + 8, PROMPT_MAX, slots=BATCH)
            decode_point(f"{tag}_decode_b8", other, BATCH, steps, lengths)
            prefill_point(f"{tag}_prefill_2048", other, PREFILL_TOKENS, 3 if dt == "bf16" else 1)
            other.close()
    out = {
        "metric": f"decode tok/s at batch 8 ({MODEL['label']} shape, random weights)", "value": round(value, 1),
        "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": max(3, args.warmup),
        "ms_per_step": round(ms_step, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": dtype, "data": "synthetic", "impl": "ours",
        "config": {
            "model": MODEL["name"], "layers": nlayers, "layers_of_model": MODEL["nlayers"], "emb_dim": MODEL["emb_dim"],
            "nheads": MODEL["nheads"], "kvheads": MODEL["kvheads"], "head_dim": MODEL["head_dim"],
            "ffn_hidden": MODEL["ffn_hidden"], "vocab": MODEL["vocab"], "context": MODEL["context"],
            "global_batch": BATCH, "seq_len": f"prompts uniform in [{PROMPT_MIN},{PROMPT_MAX}]",
            "mean_context": round(context / BATCH, 1), "prefill_tokens": PREFILL_TOKENS, "parallelism": "1 gpu",
            "weights": "random N(0,0.02), seed 0",
            "l2": f"weights read per step ({decode_bytes(nlayers, 0, MODEL, run.itemsize) / 1e9:.0f} GB) exceed L2; no flush",
            "timed": f"median of {REGIONS} regions of {args.steps} steps", "cache_block_tokens": 64,
            "peaks": pk["source"] + ("" if dtype == "bf16" else f"; fp32 arithmetic {FP32_TFLOPS_NOMINAL:.1f} TFLOP/s nominal"),
        },
        "clocks": sampler.summary(),
        "e2e": {"value": round(e2e, 1), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h},
        "gpu_launches": int(launched),
        "prefill": {"value": round(PREFILL_TOKENS / (pf_ms / 1e3), 1), "tokens": PREFILL_TOKENS, "ms": round(pf_ms, 3),
                    "frac": round(pf_frac, 4)},
        "roofline": {"bound": "hbm", "achieved": round(gbs, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(gbs / pk["hbm_gbs"], 4)},
        "regions": {"count": REGIONS, "ms_per_step": [round(x, 4) for x in per_region]},
        "points": points, "points_frac": fracs,
    }
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# --compare goletar: the Goletar design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
GOLETAR_SHAPE = dict(width=4096, recurrent_width=4096, heads=32, dim=96, rot_dim=32, vdim=128, kv_rank=512, experts=16,
                     top=4, ff=3584, vocab=128256)


def goletar_layers(kinds, with_experts=True):
    from fms_b200.models.goletar import latent_layer, mingru_layer, moe

    g = GOLETAR_SHAPE
    mlp = moe(g["experts"], g["top"], g["ff"], 7.0) if with_experts else None
    return [mingru_layer(g["recurrent_width"], mlp) if k == "mingru" else
            latent_layer(g["heads"], g["dim"], g["rot_dim"], g["vdim"], g["kv_rank"], 10000.0, mlp) for k in kinds]


def goletar_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens reads)
    of the given layers: products, attention over the cached latents, the experts each token uses (for a decode step:
    the distinct experts that `batch` tokens are expected to hit)."""
    g = GOLETAR_SHAPE
    d, flops, weights, cache = g["width"], 0.0, 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        if layer["type"] == "mingru":
            w = 4 * m["width"] * d
            att = 0.0
        else:
            h, dim, rot, v, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w = d * (h * (dim + rot) + r + rot + h) + h * dim * r + h * v * r + h * v * d
            att = tokens * tokens * h * (2 * r + rot)  # causal half of 2 T^2 (width + rank) a head
            cache += batch_context * (r + rot) * 2
        flops += 2 * tokens * w + att
        weights += 2 * w
        if layer.get("mlp"):
            e, top, f = g["experts"], g["top"], g["ff"]
            flops += 2 * tokens * (top * 3 * f * d + e * d)
            hit = e * (1 - (1 - top / e) ** batch)
            weights += 2 * (hit * 3 * f * d + e * d)
    head = 2 * g["vocab"] * d
    return flops + head, weights + head + cache


class GoletarMeasured(Measured):
    """A Goletar model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.goletar import Goletar, GoletarConfig
        from fms_b200.weights.sources import RandomSource

        g = GOLETAR_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Goletar(GoletarConfig(vocab=g["vocab"], width=g["width"], layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_goletar(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Goletar design at the width of the benchmark's Llama (alternating minGRU and latent attention,
    each with 16 experts of 3,584 of which a token takes 4: the dense feed-forward's 14,336 hidden values a token), for as
    many Llama-3-8B layers, and for each of Goletar's parts alone (models of one kind of layer, with and without
    experts).  Each figure with its fraction of the measured peak: flops of a prompt over the bf16 product peak, bytes
    a decode step reads over the copy peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "goletar", "layers": n, "shape": GOLETAR_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    kinds = ["mingru" if i % 2 == 0 else "latent_attention" for i in range(n)]
    variants = [("goletar", goletar_layers(kinds)), ("mingru_only", goletar_layers(["mingru"] * n, False)),
                ("latent_attention_only", goletar_layers(["latent_attention"] * n, False)),
                ("mingru_with_experts", goletar_layers(["mingru"] * n))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(GoletarMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: goletar_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# --compare niletar: the Niletar design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
NILETAR_SHAPE = dict(width=4096, vocab=128256, ff=14336, heads=32, kv_heads=8, dim=128, rot_dims=64,
                     delta_heads=16, delta_kv_heads=16, delta_dim=128, delta_vdim=128, rank=64,
                     ssm_heads=128, ssm_vdim=64, state=128, groups=8, conv=4)


def niletar_layers(kinds, with_mlp=True):
    from fms_b200.models.niletar import attention_side, delta_side, dense_mlp, mamba2_layer, parallel_layer

    g = NILETAR_SHAPE
    mlp = dense_mlp(g["ff"]) if with_mlp else None
    par = lambda: parallel_layer(
        attention_side(g["heads"], g["kv_heads"], g["dim"], g["dim"], g["rot_dims"], 500000.0, g["dim"] ** -0.5),
        delta_side(g["delta_heads"], g["delta_kv_heads"], g["delta_dim"], g["delta_vdim"], g["conv"], g["rank"], g["rank"]),
        0.5, 0.5, mlp)
    ssm = lambda: mamba2_layer(g["ssm_heads"], g["ssm_vdim"], g["state"], g["groups"], g["groups"], g["conv"], mlp)
    return [par() if k == "parallel" else ssm() for k in kinds]


def niletar_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens
    reads and writes) of the given layers: products, attention over the cache, the two scans (6 flops per state value
    and token for the state-space scan, 8 for the delta rule: they run in float32 on the CUDA cores), the states of the
    sequences (read and written once a step)."""
    g = NILETAR_SHAPE
    d, flops, moved = g["width"], 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        if layer["type"] == "mamba2":
            h, v, n, gr = m["heads"], m["vdim"], m["state"], m["groups"]
            inner = h * v
            w = d * (2 * inner + 2 * gr * n + h) + inner * d
            flops += 6.0 * tokens * inner * n
            moved += 2 * 4 * batch * inner * n
        else:
            l, r = m["left"], m["right"]
            w = d * (l["heads"] * l["dim"] + 2 * l["kv_heads"] * l["dim"] + l["heads"] * l["vdim"]) + l["heads"] * l["vdim"] * d
            flops += 2.0 * tokens * tokens * l["heads"] * l["dim"]  # the causal half of 4 T^2 per head and value
            moved += 2 * 2 * batch_context * l["kv_heads"] * l["dim"]
            rk = r.get("decay_rank", 0) + r.get("gate_rank", 0)
            w += d * (2 * r["kv_heads"] * r["dim"] + r["heads"] * r["vdim"] + r["heads"] + rk) + r["heads"] * r["vdim"] * d
            w += r["decay_rank"] * r["heads"] * r["dim"] + r["gate_rank"] * r["heads"] * r["vdim"]
            flops += 8.0 * tokens * r["heads"] * r["dim"] * r["vdim"]
            moved += 2 * 4 * batch * r["heads"] * r["dim"] * r["vdim"]
        if layer.get("mlp"):
            w += 3 * layer["mlp"]["ff"] * d
        flops += 2.0 * tokens * w
        moved += 2 * w
    head = 2 * g["vocab"] * d
    return flops + head, moved + head


class NiletarMeasured(Measured):
    """A Niletar model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.niletar import Niletar, NiletarConfig
        from fms_b200.weights.sources import RandomSource

        g = NILETAR_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Niletar(NiletarConfig(vocab=g["vocab"], width=g["width"], postln_alpha=2.0, layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_niletar(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Niletar design at the width of the benchmark's Llama (alternating the parallel mixer and the
    state-space scan, each with the dense feed-forward of 14,336), for as many Llama-3-8B layers, and for each of
    Niletar's mixers alone (models of one kind of layer without a feed-forward).  Each figure with its fraction of the
    measured peak: flops of a prompt over the bf16 product peak, bytes a decode step moves over the copy peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "niletar", "layers": n, "shape": NILETAR_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    kinds = ["parallel" if i % 2 == 0 else "mamba2" for i in range(n)]
    variants = [("niletar", niletar_layers(kinds)), ("parallel_only", niletar_layers(["parallel"] * n, False)),
                ("mamba2_only", niletar_layers(["mamba2"] * n, False))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(NiletarMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: niletar_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# --compare figonex: the Figonex design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
FIGONEX_SHAPE = dict(width=4096, vocab=128256, ff=14336, heads=32, kv_heads=8, dim=128, rot_dims=64,
                     memory_heads=32, memory_dim=128, memory_vdim=128, gate_cap=15.0)


def figonex_layers(kinds, with_mlp=True):
    from fms_b200.models.figonex import attention_layer, dense_mlp, lightning_layer, mlstm_layer

    g = FIGONEX_SHAPE
    mlp = dense_mlp(g["ff"]) if with_mlp else None
    h = g["memory_heads"]
    decays = [1.0 - 0.1 * 0.01 ** (i / max(1, h - 1)) for i in range(h)]
    make = {"mlstm": lambda: mlstm_layer(h, g["memory_dim"], g["memory_vdim"], g["gate_cap"], mlp),
            "attention": lambda: attention_layer(g["heads"], g["kv_heads"], g["dim"], g["rot_dims"], 500000.0, None,
                                                 g["dim"] ** -0.5, mlp),
            "lightning": lambda: lightning_layer(h, g["memory_dim"], g["memory_vdim"], decays, mlp)}
    return [make[k]() for k in kinds]


def figonex_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens
    reads and writes) of the given layers: products, attention over the cache (keys and values are cached apart: a
    value is its key before norm and rotation), the scans of the matrix memories (6 flops per state value and token:
    they run in float32 on the CUDA cores), the states of the sequences (read and written once a step)."""
    g = FIGONEX_SHAPE
    d, flops, moved = g["width"], 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        h, k = m["heads"], m["dim"]
        if layer["type"] == "attention":
            w = d * (h * k + m["kv_heads"] * k + h) + h * k * d
            flops += 2.0 * tokens * tokens * h * k  # the causal half of 4 T^2 per head and value
            moved += 2 * 2 * batch_context * m["kv_heads"] * k
        else:
            v = m["vdim"]
            w = d * (2 * h * k + 2 * h * v + (2 * h if layer["type"] == "mlstm" else 0)) + h * v * d
            flops += 6.0 * tokens * h * k * v
            moved += 2 * 4 * batch * h * k * v
        if layer.get("mlp"):
            w += 3 * layer["mlp"]["ff"] * d
        flops += 2.0 * tokens * w
        moved += 2 * w
    head = 2 * g["vocab"] * d
    return flops + head, moved + head


class FigonexMeasured(Measured):
    """A Figonex model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.figonex import Figonex, FigonexConfig
        from fms_b200.weights.sources import RandomSource

        g = FIGONEX_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Figonex(FigonexConfig(vocab=g["vocab"], width=g["width"], embedding_scale=8.0, layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_figonex(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Figonex design at the width of the benchmark's Llama (a gated matrix memory, attention,
    attention, a decaying matrix memory, each with the dense feed-forward of 14,336), for as many Llama-3-8B layers, and
    for each of Figonex's mixers alone (models of one kind of layer without a feed-forward).  Each figure with its
    fraction of the measured peak: flops of a prompt over the bf16 product peak, bytes a decode step moves over the copy
    peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "figonex", "layers": n, "shape": FIGONEX_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    order = ("mlstm", "attention", "attention", "lightning")
    variants = [("figonex", figonex_layers([order[i % 4] for i in range(n)])),
                ("mlstm_only", figonex_layers(["mlstm"] * n, False)),
                ("attention_only", figonex_layers(["attention"] * n, False)),
                ("lightning_only", figonex_layers(["lightning"] * n, False))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(FigonexMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: figonex_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# the reference, unmodified, through its own public API
# --------------------------------------------------------------------------------------------------
def run_reference(args):
    ref = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isdir(os.path.join(ref, "fms")):
        print(json.dumps({"impl": "reference", "unavailable": "baseline/_ref holds no installed reference"}))
        return
    sys.path.insert(0, ref)
    try:
        import torch
        from fms.models import get_model
        from fms.utils.generation import generate, pad_input_ids
    except Exception as e:  # noqa: BLE001
        print(json.dumps({"impl": "reference", "unavailable": f"import failed: {type(e).__name__}: {e}"[:200]}))
        return

    nlayers = args.layers or MODEL["nlayers"]
    torch.manual_seed(0)
    model = get_model("llama", MODEL["variant"], device_type="cuda", data_type=torch.bfloat16, nlayers=nlayers)
    model.eval()
    torch.set_grad_enabled(False)
    warmup = max(3, args.warmup)

    def decode(batch, steps):
        lengths = prompt_lengths(batch)
        prompts = [torch.tensor(p, dtype=torch.long, device="cuda") for p in random_prompts(lengths, MODEL["vocab"])]
        ids, extra = pad_input_ids(prompts)
        extra["last_n_tokens"] = 1
        events = []

        def hook(i, logits, next_val, kwargs):
            ev = torch.cuda.Event(enable_timing=True)
            ev.record()
            events.append(ev)
            return next_val, kwargs

        _, times = generate(model, ids, max_new_tokens=1 + warmup + steps, use_cache=True, do_sample=False,
                            timing="per-token", post_iteration_hook=hook, extra_kwargs=extra)
        torch.cuda.synchronize()
        ms = events[-steps - 1].elapsed_time(events[-1])
        context = sum(lengths) + batch * (1 + warmup + steps / 2.0)
        return batch * steps / (ms / 1e3), ms / steps, batch * steps / sum(times[-steps:]), context

    sampler = ClockSampler()
    sampler.start()
    value, ms_step, e2e, context = decode(BATCH, args.steps)
    sampler.stop()
    side = max(32, args.steps // 2)
    b1 = decode(1, side)[0]
    b64 = decode(64, side)[0]
    ids = torch.tensor(random_prompts([PREFILL_TOKENS], MODEL["vocab"], seed=7), dtype=torch.long, device="cuda")
    ms = []
    for i in range(8):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        model(ids, use_cache=True, last_n_tokens=1)
        end.record()
        torch.cuda.synchronize()
        if i >= 3:
            ms.append(start.elapsed_time(end))
    pf_ms = statistics.median(ms)
    pk = peaks()
    gbs = decode_bytes(nlayers, context) / (ms_step / 1e3) / 1e9
    print(json.dumps({
        "metric": f"decode tok/s at batch 8 ({MODEL['label']} shape, random weights)", "value": round(value, 1),
        "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup, "ms_per_step": round(ms_step, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "impl": "reference",
        "config": {"model": MODEL["name"], "layers": nlayers, "layers_of_model": MODEL["nlayers"], "global_batch": BATCH,
                   "seq_len": f"prompts uniform in [{PROMPT_MIN},{PROMPT_MAX}], left-padded", "parallelism": "1 gpu",
                   "path": "fms get_model + generate, eager, sdpa, use_cache", "prefill_tokens": PREFILL_TOKENS},
        "clocks": sampler.summary(),
        "e2e": {"value": round(e2e, 1), "unit": "tok/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "prefill": {"value": round(PREFILL_TOKENS / (pf_ms / 1e3), 1), "tokens": PREFILL_TOKENS, "ms": round(pf_ms, 3),
                    "frac": round(prefill_flops(nlayers, PREFILL_TOKENS) / (pf_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(gbs, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(gbs / pk["hbm_gbs"], 4)},
        "points": {"decode_b1": round(b1, 1), "decode_b64": round(b64, 1)},
    }))


# --------------------------------------------------------------------------------------------------
# --compare giganex: the Giganex design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
GIGANEX_SHAPE = dict(width=4096, vocab=128256, groups=8, ff=14336, experts=16, top=4, expert_ff=3584,
                     heads=32, kv_heads=8, dim=128, rot_dims=128, chunk=8192, softcap=30.0,
                     delta_heads=16, delta_kv_heads=16, delta_dim=128, delta_vdim=128, conv=4,
                     latent_heads=32, latent_dim=96, latent_rot=32, latent_vdim=128, q_rank=1536, kv_rank=512, window=4096)
_GIGANEX_STRETCH = {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}


def giganex_layers(kinds, mlps):
    """`kinds`: the mixers ("parallel", "latent_attention", "attention"), `mlps`: their feed-forwards ("dense", "moe", None)."""
    from fms_b200.models.giganex import (attention_layer, capped_side, delta_side, dense_mlp, latent_layer, moe_mlp,
                                         parallel_layer, rotation)

    g = GIGANEX_SHAPE
    out = []
    for kind, which in zip(kinds, mlps):
        mlp = None if which is None else (dense_mlp(g["ff"]) if which == "dense" else moe_mlp(g["experts"], g["top"], g["expert_ff"], 2.0))
        if kind == "parallel":
            out.append(parallel_layer(capped_side(g["heads"], g["kv_heads"], g["dim"], g["dim"], g["dim"] ** -0.5, g["softcap"]),
                                      delta_side(g["delta_heads"], g["delta_kv_heads"], g["delta_dim"], g["delta_vdim"], g["conv"]),
                                      0.5, 0.5, mlp))
        elif kind == "latent_attention":
            out.append(latent_layer(g["latent_heads"], g["latent_dim"], g["latent_rot"], g["latent_vdim"], g["q_rank"], g["kv_rank"],
                                    10000.0, _GIGANEX_STRETCH, (g["latent_dim"] + g["latent_rot"]) ** -0.5, g["window"], mlp))
        else:
            out.append(attention_layer(g["heads"], g["kv_heads"], g["dim"], g["dim"], rotation(g["rot_dims"], 500000.0, _GIGANEX_STRETCH),
                                       g["dim"] ** -0.5, g["chunk"], mlp))
    return out


def giganex_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens
    reads and writes) of the given layers: products, attention over the cache (keys and values, or latents), the delta
    rule (8 flops per state value and token, float32 on the CUDA cores; its states read and written once a step), the
    experts each token uses (for a decode step: the distinct experts that `batch` tokens are expected to hit)."""
    g = GIGANEX_SHAPE
    d, flops, moved = g["width"], 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        if layer["type"] == "attention":
            w = d * (m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"])) + m["heads"] * m["vdim"] * d
            flops += tokens * tokens * m["heads"] * (m["dim"] + m["vdim"])  # the causal half of 2 T^2 (dim + vdim) a head
            moved += 2 * batch_context * m["kv_heads"] * (m["dim"] + m["vdim"])
        elif layer["type"] == "latent_attention":
            h, dim, rot, v, qr, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            w = d * (qr + r + rot) + qr * h * (dim + rot) + h * dim * r + h * v * r + h * v * d
            flops += tokens * tokens * h * (2 * r + rot)
            moved += 2 * batch_context * (r + rot)
        else:
            l, r = m["left"], m["right"]
            w = d * (l["heads"] * l["dim"] + l["kv_heads"] * (l["dim"] + l["vdim"]) + l["heads"] * l["vdim"]) + l["heads"] * l["vdim"] * d
            flops += tokens * tokens * l["heads"] * (l["dim"] + l["vdim"])
            moved += 2 * batch_context * l["kv_heads"] * (l["dim"] + l["vdim"])
            w += d * (2 * r["kv_heads"] * r["dim"] + 2 * r["heads"] * r["vdim"] + 2 * r["heads"]) + r["heads"] * r["vdim"] * d
            flops += 8.0 * tokens * r["heads"] * r["dim"] * r["vdim"]
            moved += 2 * 4 * batch * r["heads"] * r["dim"] * r["vdim"]
        flops += 2.0 * tokens * w
        moved += 2 * w
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] == "dense":
            flops += 2.0 * tokens * 3 * mlp["ff"] * d
            moved += 2 * 3 * mlp["ff"] * d
        elif mlp:
            e, top, f = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            flops += 2.0 * tokens * (top * 2 * f * d + e * d)
            hit = e * (1 - (1 - top / e) ** batch)
            moved += 2 * (hit * 2 * f * d + e * d)
    head = 2 * g["vocab"] * d
    return flops + head, moved + head


class GiganexMeasured(Measured):
    """A Giganex model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.giganex import Giganex, GiganexConfig
        from fms_b200.weights.sources import RandomSource

        g = GIGANEX_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Giganex(GiganexConfig(vocab=g["vocab"], width=g["width"], norm_groups=g["groups"], layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_giganex(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Giganex design at the width of the benchmark's Llama (the two mixers side by side with the dense
    feed-forward of 14,336, attention over latents and attention over runs each with 16 experts of 3,584 of which a token
    takes 4, taking turns), for as many Llama-3-8B layers, and for each of Giganex's mixers alone (models of one kind of
    layer without a feed-forward) and the experts under one of them.  Each figure with its fraction of the measured
    peak: flops of a prompt over the bf16 product peak, bytes a decode step moves over the copy peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "giganex", "layers": n, "shape": GIGANEX_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    order = [("parallel", "dense"), ("latent_attention", "moe"), ("attention", "moe")]
    mixed = [order[i % 3] for i in range(n)]
    variants = [("giganex", giganex_layers([k for k, _ in mixed], [f for _, f in mixed])),
                ("parallel_only", giganex_layers(["parallel"] * n, [None] * n)),
                ("latent_attention_only", giganex_layers(["latent_attention"] * n, [None] * n)),
                ("attention_only", giganex_layers(["attention"] * n, [None] * n)),
                ("attention_with_experts", giganex_layers(["attention"] * n, ["moe"] * n))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(GiganexMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: giganex_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# --compare bolinex: the Bolinex design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
BOLINEX_SHAPE = dict(width=4096, vocab=128256, ff=14336, experts=16, top=4, groups=4, keep=2, expert_ff=3584, shared_ff=3584,
                     heads=32, kv_heads=8, dim=128, vdim=128, window=4096, softcap=30.0, side_dim=256, max_positions=8192)


def bolinex_layers(mlps):
    """`mlps`: the layers' feed-forwards ("dense", "moe", None)."""
    from fms_b200.models.bolinex import attention_layer, dense_mlp, moe_mlp

    g = BOLINEX_SHAPE
    make = {None: lambda: None, "dense": lambda: dense_mlp(g["ff"]),
            "moe": lambda: moe_mlp(g["experts"], g["top"], g["expert_ff"], g["shared_ff"], g["groups"], g["keep"])}
    return [attention_layer(g["heads"], g["kv_heads"], g["dim"], g["vdim"], g["dim"] ** -0.5, g["softcap"], g["window"], True,
                            make[which]()) for which in mlps]


def bolinex_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens
    reads and writes) of the given layers: products, attention over the cache, the token side's two small products, the
    experts each token uses (for a decode step: the distinct experts that `batch` tokens are expected to hit)."""
    g = BOLINEX_SHAPE
    d, flops, moved = g["width"], 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        h, kv, k, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w = d * (h * k + kv * (k + v) + h * v) + h * v * d + 2 * d * g["side_dim"]
        flops += tokens * tokens * h * (k + v)  # the causal half of 2 T^2 (dim + vdim) a head
        moved += 2 * batch_context * kv * (k + v)
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] == "dense":
            w += 2 * mlp["ff"] * d
        elif mlp:
            e, top, f = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            w += 3 * mlp["shared"]["ff"] * d + e * d
            flops += 2.0 * tokens * top * 3 * f * d
            moved += 2 * e * (1 - (1 - top / e) ** batch) * 3 * f * d
        flops += 2.0 * tokens * w
        moved += 2 * w
    head = 2 * g["vocab"] * d
    return flops + head, moved + head


class BolinexMeasured(Measured):
    """A Bolinex model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.bolinex import Bolinex, BolinexConfig
        from fms_b200.weights.sources import RandomSource

        g = BOLINEX_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Bolinex(BolinexConfig(vocab=g["vocab"], width=g["width"], side_dim=g["side_dim"],
                                           max_positions=g["max_positions"], layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_bolinex(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Bolinex design at the width of the benchmark's Llama (layers with the dense feed-forward of 14,336
    and layers with 16 experts of 3,584 of which a token takes 4, beside a shared one, taking turns), for as many
    Llama-3-8B layers, and for each kind of layer alone (the mixer without a feed-forward, with the dense one, with the
    experts).  Each figure with its fraction of the measured peak: flops of a prompt over the bf16 product peak, bytes a
    decode step moves over the copy peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "bolinex", "layers": n, "shape": BOLINEX_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    variants = [("bolinex", bolinex_layers([("dense", "moe")[i % 2] for i in range(n)])),
                ("attention_only", bolinex_layers([None] * n)),
                ("attention_with_dense", bolinex_layers(["dense"] * n)),
                ("attention_with_experts", bolinex_layers(["moe"] * n))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(BolinexMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: bolinex_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
# --compare tabatar: the Tabatar design beside Llama at equal width, layer for layer
# --------------------------------------------------------------------------------------------------
TABATAR_SHAPE = dict(width=4096, vocab=128256, streams=2, ff=14336, experts=16, top=4, expert_ff=3584, shared_ff=3584, heads=32,
                     kv_heads=8, dim=128, vdim=128, window=4096, gla_heads=32, gla_dim=128, gla_vdim=128, tau=16.0, rank=16,
                     softcap=30.0)


def tabatar_layers(kinds, mlps):
    """`kinds`: the mixers ("attention", "gla"), `mlps`: their feed-forwards ("dense", "moe", None)."""
    from fms_b200.models.tabatar import attention_layer, dense_mlp, gla_layer, moe_mlp

    g = TABATAR_SHAPE
    rot = {"base": 500000.0, "dims": g["dim"], "scaling": {"factor": 8.0, "high": 4.0, "low": 1.0, "original": 8192}}
    out = []
    for kind, which in zip(kinds, mlps):
        mlp = {None: lambda: None, "dense": lambda: dense_mlp(g["ff"]),
               "moe": lambda: moe_mlp(g["experts"], g["top"], g["expert_ff"], g["shared_ff"])}[which]()
        out.append(attention_layer(g["heads"], g["kv_heads"], g["dim"], g["vdim"], g["dim"] ** -0.5, g["window"], rot, mlp)
                   if kind == "attention" else gla_layer(g["gla_heads"], g["gla_dim"], g["gla_vdim"], g["tau"], g["rank"], mlp))
    return out


def tabatar_counts(layers, tokens, batch_context, batch):
    """(flops of a prompt of `tokens`, bytes a decode step of `batch` sequences with `batch_context` cached tokens
    reads and writes) of the given layers: products, attention over the cache, the matrix memories (6 flops per state value
    and token, float32 on the CUDA cores; the states read and written once a step), the experts each token uses (for a
    decode step: the distinct experts that `batch` tokens are expected to hit)."""
    g = TABATAR_SHAPE
    d, flops, moved = g["width"], 0.0, 0.0
    for layer in layers:
        m = layer["mixer"]
        h, k, v = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            kv = m["kv_heads"]
            w = d * (h * k + kv * (k + v) + h * v) + h * v * d
            flops += tokens * tokens * h * (k + v)  # the causal half of 2 T^2 (dim + vdim) a head
            moved += 2 * batch_context * kv * (k + v)
        else:
            w = d * (2 * h * k + 2 * h * v + m["rank"]) + m["rank"] * h * k + h * v * d
            flops += 6.0 * tokens * h * k * v
            moved += 2 * 4 * batch * h * k * v
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] == "dense":
            w += 2 * mlp["ff"] * d
        elif mlp:
            e, top, f = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            w += 3 * mlp["shared"]["ff"] * d + (e + 1) * d
            flops += 2.0 * tokens * top * 3 * f * d
            moved += 2 * e * (1 - (1 - top / e) ** batch) * 3 * f * d
        flops += 2.0 * tokens * w
        moved += 2 * w
    head = 2 * g["vocab"] * d
    return flops + head, moved + head


class TabatarMeasured(Measured):
    """A Tabatar model of given layers on the device, measured like the Llama one."""

    def __init__(self, layers, room, max_prompt, slots):
        import torch

        from fms_b200.models.tabatar import Tabatar, TabatarConfig
        from fms_b200.weights.sources import RandomSource

        g = TABATAR_SHAPE
        self.m, self.dtype, self.nlayers, self.itemsize, self.layers = dict(vocab=g["vocab"]), "bf16", len(layers), 2, layers
        self.model = Tabatar(TabatarConfig(vocab=g["vocab"], width=g["width"], embedding_scale=g["width"] ** 0.5, streams=g["streams"],
                                           logit_softcap=g["softcap"], layers=layers))
        self.model.load(RandomSource(self.model.checkpoint_layout(), 0, dtype=torch.bfloat16, device="cuda"), "native", "cuda",
                        torch.bfloat16)
        self.engine = self.model.new_engine(max_tokens=slots * (max_prompt + 2 * room + 128), max_slots=slots)
        self.torch = torch


def run_tabatar(args):
    """One JSON line: prompts of 512 and 2,048 tokens and decode steps of 1, 8 and 64 sequences, for `--layers` layers
    (default 4) of the Tabatar design at the width of the benchmark's Llama (attention with the dense feed-forward of 14,336
    and gated linear attention of 32 heads of 128 x 128 with 16 experts of 3,584 of which a token takes 4, beside a shared one,
    taking turns, between two residual streams), for as many Llama-3-8B layers, for each mixer alone, and for each
    feed-forward under attention.  Each figure with its fraction of the measured peak: flops of a prompt over the bf16
    product peak, bytes a decode step moves over the copy peak."""
    pk = peaks()
    n = args.layers or 4
    steps, warm = max(16, args.steps // 2), max(3, args.warmup // 2)
    room = warm + 3 * steps + 8
    lengths = {1: [1024], 8: [1024] * 8, 64: [1024] * 64}
    out = {"compare": "tabatar", "layers": n, "shape": TABATAR_SHAPE, "peaks": pk, "steps": steps, "warmup": warm, "models": {}}

    def measure(run, name, flops_bytes):
        row = {}
        for tokens in (512, 2048):
            ms = run.prefill(tokens, 3)
            row[f"prefill_{tokens}"] = {"ms": round(ms, 3), "tok_s": round(tokens / (ms / 1e3), 1),
                                        "frac_of_bf16_peak": round(flops_bytes(tokens, 0, 0)[0] / (ms / 1e3) / 1e12 / pk["bf16_tflops"], 4)}
        for b in (1, 8, 64):
            v, ms, ctx, _, _ = run.device_decode(b, steps, warm, lengths[b], regions=3)
            row[f"decode_b{b}"] = {"ms": round(ms, 4), "tok_s": round(v, 1),
                                   "frac_of_copy_peak": round(flops_bytes(0, ctx, b)[1] / (ms / 1e3) / 1e9 / pk["hbm_gbs"], 4)}
        out["models"][name] = row
        run.close()

    mixed = [("attention", "dense"), ("gla", "moe")]
    variants = [("tabatar", tabatar_layers([mixed[i % 2][0] for i in range(n)], [mixed[i % 2][1] for i in range(n)])),
                ("attention_only", tabatar_layers(["attention"] * n, [None] * n)),
                ("gla_only", tabatar_layers(["gla"] * n, [None] * n)),
                ("attention_with_dense", tabatar_layers(["attention"] * n, ["dense"] * n)),
                ("attention_with_experts", tabatar_layers(["attention"] * n, ["moe"] * n))]
    if args.only:
        variants = [v for v in variants if v[0] == args.only]
    for name, layers in variants:
        measure(TabatarMeasured(layers, room, 2048, 64), name,
                lambda tokens, ctx, b, layers=layers: tabatar_counts(layers, tokens, ctx, b))
    if not args.only or args.only == "llama":
        llama = Measured(MODEL, "bf16", n, room, 2048, slots=64)
        measure(llama, "llama", lambda tokens, ctx, b: (prefill_flops(n, tokens), decode_bytes(n, ctx)))
    print(json.dumps(out))


# --------------------------------------------------------------------------------------------------
def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--gpus", type=int, default=int(os.environ.get("WORLD_SIZE", "1")))
    ap.add_argument("--steps", type=int, default=64)
    # the default covers the 20 or so steps (80 ms) that the GPU's clocks take to come back up after the prefill
    ap.add_argument("--warmup", type=int, default=24)
    ap.add_argument("--impl", choices=["ours", "reference"], default="ours")
    ap.add_argument("--only", default="", help="decode_b<batch> or prefill: run and print that part only; gemm_rows, "
                    "attention_prefill, attention_decode: single kernels over a range of sizes")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the model has (named in config)")
    ap.add_argument("--model", choices=sorted(MODELS), default="llama-3-8b",
                    help="the shape to measure; the default is the benchmark's, the others are its further configurations")
    ap.add_argument("--dtype", choices=["bf16", "fp32"], default="bf16", help="fp32: the true 32-bit path")
    ap.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS, help="with --only prefill: the prompt's length")
    ap.add_argument("--points", choices=["default", "main", "long"], default="default",
                    help="main: without the further configurations; long: also decode at batch 64 with 8k contexts")
    ap.add_argument("--compare", choices=["", "goletar", "niletar", "figonex", "giganex", "bolinex", "tabatar"], default="",
                    help="goletar: the Goletar design beside as many Llama layers of equal width (--layers, default 4; "
                    "--only goletar|mingru_only|latent_attention_only|mingru_with_experts|llama for one of them); "
                    "niletar: the Niletar design likewise (--only niletar|parallel_only|mamba2_only|llama); "
                    "figonex: the Figonex design likewise (--only figonex|mlstm_only|attention_only|lightning_only|llama); "
                    "giganex: the Giganex design likewise (--only giganex|parallel_only|latent_attention_only|attention_only|"
                    "attention_with_experts|llama); "
                    "bolinex: the Bolinex design likewise (--only bolinex|attention_only|attention_with_dense|"
                    "attention_with_experts|llama); "
                    "tabatar: the Tabatar design likewise (--only tabatar|attention_only|gla_only|attention_with_dense|"
                    "attention_with_experts|llama)")
    args = ap.parse_args()
    choose_model(args.model)
    if args.gpus != 1:
        if int(os.environ.get("RANK", "0")) == 0:
            print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not measured")
        sys.exit(2)
    if args.compare == "goletar":
        run_goletar(args)
    elif args.compare == "niletar":
        run_niletar(args)
    elif args.compare == "figonex":
        run_figonex(args)
    elif args.compare == "giganex":
        run_giganex(args)
    elif args.compare == "bolinex":
        run_bolinex(args)
    elif args.compare == "tabatar":
        run_tabatar(args)
    elif args.impl == "reference":
        run_reference(args)
    elif args.only in ("gemm_rows", "attention_prefill", "attention_decode"):
        run_kernels(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
