"""Decode and prefill throughput of the engine at Qwen3 layer sizes, one GPU.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]
                    [--shape 8b|14b|32b] [--workload decode|mixed]
    python bench.py --design nekedra|tonanex|pabalorn|dovorax|lokizen|mapovik [--design-size 2048|4096]

A "step" is one decode step: every request of the batch gets its next token.
The default run has the sizes of the 8B configuration (36 layers, hidden 4096,
32/8 heads of 128, intermediate 12288, vocabulary 151936), random weights in
bfloat16, a batch of 8 and 2,048 tokens of context per request.  It prints one
JSON line:

* ``value``: decoded tokens a second of whole steps run back to back through the
  step function (host half -- checks, page reservation, batch layout -- and
  device half -- one upload, the forward), timed on the device with CUDA events
  around blocks of exactly ``--steps`` steps; the block is repeated until at
  least two seconds are timed and the median block is reported.
  ``device_half_ms`` is the device half alone (the host half done before the
  first event), ``eager_ms`` the same step launched kernel by kernel instead of
  replayed from its CUDA graph.
* ``e2e``: the same through the Python entry point (``LLM.step``), by the wall
  clock, host token ids in and sampled token ids out every step.
* ``prefill``: a 2,048-token prompt (median of runs back to back: the GPU is at
  its power cap by then); ``roofline``: the decode step's bytes over its time
  against the measured copy bandwidth; ``points``: decode at batch 1 and 64,
  device-timed and end to end; ``kernels``: a table of where an eager decode
  step's and a prefill's time goes, kernel by kernel.

``--shape 32b`` runs the 32B configuration's workload (decode at batch 1 and 64
with 4,096 tokens of context, one 2,048-token prefill), ``--shape 14b`` (whose
default workload is ``mixed``) 32 requests with prompts of 128 to 3,072 tokens
prefilled in portions of up to 512 tokens beside the decoding ones, through the
scheduler.

``--design nekedra`` leaves all of that aside and prints another line: prefill
and decode of four-layer Nekedra stacks (each mixer alone, and mixed) beside the
Qwen3 decoder at equal width, heads and feed-forward size, with the kernels an
eager step spends its time in (``run_design``).
``--design tonanex`` does the same for Tonanex stacks with a dense feed-forward
and with routed experts, ``--design pabalorn`` for Pabalorn stacks of attention
layers, of layers with an attention and a selective scan side by side, and of
both in turn, beside Qwen3 and the Tonanex stack with routed experts,
``--design dovorax`` for Dovorax stacks of each of its three layer kinds and of
all of them, beside Qwen3, Nekedra's latent attention and delta rule, and the
Tonanex stack with routed experts, ``--design lokizen`` for Lokizen stacks of
attention, of retention and of both in a loop, ``--design mapovik`` for Mapovik
stacks of delta-rule layers, of layers with an attention and a state space side
by side, and of both in a loop, beside Nekedra's delta rule, Tonanex's routed
experts and Pabalorn's side-by-side layers.
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

BASE = {"architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "head_dim": 128, "num_key_value_heads": 8,
        "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": False,
        "max_position_embeddings": 8192}   # room for the tokens decoded on top of a 4,096-token context
SHAPES = {      # layer sizes of the benchmark configurations; context = tokens each request holds while decoding
    "8b": dict(BASE, num_hidden_layers=36, hidden_size=4096, num_attention_heads=32, intermediate_size=12288),
    "14b": dict(BASE, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408),
    "32b": dict(BASE, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, intermediate_size=25600),
}
CONTEXT = {"8b": 2048, "14b": 2048, "32b": 4096}
BATCH = {"8b": 8, "14b": 8, "32b": 64}
PREFILL_TOKENS = 2048
PAGE_SIZE = 16
MIN_TIMED_SECONDS = 2.0
MAX_GROWTH = 640          # tokens a request's context may grow by over all timed blocks of one measurement


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    out = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}
    if os.path.isfile(path):
        try:
            with open(path) as f:
                got = json.load(f)
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                if isinstance(got.get(k), (int, float)) and got[k] > 0:
                    out[k] = float(got[k])
            out["source"] = "measured"
        except (OSError, ValueError):
            pass
    return out


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    NAMES = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")

    def __init__(self, index: int = 0):
        self.rows, self.proc, self.index = [], None, index

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) == 6 and parts[0].isdigit():
                self.rows.append(parts)

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        if not self.rows:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["unsampled"]}
        reasons = [n for i, n in enumerate(self.NAMES) if any(r[2 + i] == "Active" for r in self.rows)]
        return {"sm_mhz": int(statistics.median(int(r[0]) for r in self.rows)),
                "sm_max_mhz": int(self.rows[0][1]), "reasons": reasons, "samples": len(self.rows)}


def reference_arm():
    # The reference is a Rust crate; this machine has no cargo/rustc and no network, and pip cannot
    # install a crate.  Its only CUDA code (one naive linear kernel) was never wired to a model run.
    print(json.dumps({"impl": "reference", "unavailable":
                      "the reference is a Rust crate (no Python package to pip-install; no cargo/rustc here)"}))
    return 0


def build_engine(config: dict, layers: int, max_requests: int, tokens_in_cache: int, max_batch_tokens: int,
                 graphs=True):
    import torch
    from safetyraise_lmengine_b200 import Engine, spec_from_config
    from safetyraise_lmengine_b200.parts.model import tensor_decls
    from safetyraise_lmengine_b200.weights.random_init import RandomWeights
    cfg = dict(config, num_hidden_layers=layers) if "num_hidden_layers" in config else dict(config)
    spec = spec_from_config(cfg)
    src = RandomWeights(tensor_decls(spec), seed=0, device="cuda:0")
    num_pages = (tokens_in_cache + PAGE_SIZE - 1) // PAGE_SIZE + max_requests
    eng = Engine.from_source(cfg, src, dtype="bfloat16", page_size=PAGE_SIZE, num_pages=num_pages,
                             max_requests=max_requests, max_batch_tokens=max_batch_tokens, max_context=8192,
                             options={"cuda_graphs": graphs})
    torch.cuda.synchronize()
    return eng


def randomize_cache(eng):
    """Random cache contents, N(0, 1).  The work does not depend on the values, the power does: at its power cap
    the GPU runs a 32B decode step of batch 64 in 23.4 ms over such contents and in 22.2 ms over zeros."""
    pools = list(eng.cache.kv_pools.values()) + list(eng.cache.k_pools.values()) + list(eng.cache.v_pools.values())
    for pool in pools:
        flat = pool.view(-1)
        step = 1 << 26
        for lo in range(0, flat.numel(), step):
            flat[lo:lo + step].normal_(0.0, 1.0)


def fill_contexts(eng, batch: int, context: int):
    """Opens `batch` requests that each hold `context` tokens; the page accounting is the real one."""
    import torch
    slots = []
    for _ in range(batch):
        s = eng.open_request()
        assert eng.cache.reserve(s, context)
        eng.cache.commit(s, context)
        slots.append(s)
    torch.cuda.synchronize()
    return slots


def rewind(eng, slots, length: int) -> None:
    """The contexts back to `length` tokens each, where the cache can: a group with a window has given back the pages
    behind it, and its contexts stay as long as they have grown (the pool has room for that growth)."""
    for s in slots:
        try:
            eng.cache.truncate(s, length)
        except ValueError:
            pass


def blocks_for(steps: int, warmup: int, ms_per_step: float, min_seconds: float) -> int:
    """How many blocks of `steps` steps: enough for `min_seconds`, within the growth a context is allowed."""
    want = math.ceil(min_seconds * 1000.0 / max(ms_per_step * steps, 1e-3))
    return max(1, min(want, (MAX_GROWTH - warmup - 8) // max(steps, 1)))


def time_decode(eng, slots, context: int, steps: int, warmup: int, min_seconds: float):
    """Whole decode steps back to back through the step function, CUDA events around blocks of exactly
    `steps` steps.  Returns a dict: ms_per_step (median block), device_half_ms (median step, host half
    outside the events), blocks, mean_context (of the timed steps), launches (of one block)."""
    import torch
    from safetyraise_lmengine_b200 import StepEntry
    from safetyraise_lmengine_b200.kernels import ops
    gen = torch.Generator().manual_seed(0)
    vocab = eng.spec.vocab_size
    def entries():
        toks = torch.randint(0, vocab, (len(slots),), generator=gen).tolist()
        return [StepEntry(s, [t], [0]) for s, t in zip(slots, toks)]
    for _ in range(warmup):
        eng.run(eng.prepare(entries()))
    torch.cuda.synchronize()
    # the device half alone: host half before the first event
    half = []
    for _ in range(min(steps, 20)):
        prep = eng.prepare(entries())
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        eng.run(prep)
        b.record()
        torch.cuda.synchronize()
        half.append(a.elapsed_time(b))
    rewind(eng, slots, context + warmup)
    nblocks = blocks_for(steps, warmup, statistics.median(half), min_seconds)
    block_ms, launches = [], 0
    for _ in range(nblocks):
        batches = [entries() for _ in range(steps)]
        before = ops.launches
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        for e in batches:
            eng.run(eng.prepare(e))             # host half and device half of every step inside the events
        b.record()
        torch.cuda.synchronize()
        block_ms.append(a.elapsed_time(b))
        launches = ops.launches - before
    grown = warmup + nblocks * steps
    rewind(eng, slots, context)
    return {"ms_per_step": statistics.median(block_ms) / steps, "device_half_ms": statistics.median(half),
            "blocks": nblocks, "mean_context": context + warmup + (grown - warmup) // 2, "launches": launches,
            "timed_seconds": sum(block_ms) / 1000.0}


def decode_bytes(eng, batch: int, context: int) -> int:
    """Bytes a decode step has to read: every weight it uses once (the embedding table is only
    gathered) and the cache of the live requests."""
    spec = eng.spec
    total = eng.model.weight_bytes()
    if not spec.tie_word_embeddings:
        total -= spec.vocab_size * spec.hidden_size * 2      # embedding table: `batch` rows only
    total += batch * spec.hidden_size * 2
    total += batch * context * eng.cache.bytes_per_page() // eng.cache.page_size
    return total


def linear_flops_per_token(spec) -> float:
    total = 0.0
    for step in spec.run_order:
        layer = spec.layers[step.layer]
        m, ff, H = layer.mixer, layer.feed_forward, spec.hidden_size
        total += 2 * ((m.heads + 2 * m.kv_heads) * m.head_dim * H + m.heads * m.head_dim * H
                      + 3 * H * ff.intermediate_size)
    return total


def attention_flops(spec, q_len: int, start: int) -> float:
    """QK^T and PV of q_len queries that follow `start` cached tokens (causal)."""
    total = 0.0
    keys = q_len * start + q_len * (q_len + 1) / 2.0
    for step in spec.run_order:
        m = spec.layers[step.layer].mixer
        total += 2 * 2 * keys * m.heads * m.head_dim
    return total


def prefill_flops(spec, tokens: int) -> float:
    return tokens * linear_flops_per_token(spec) + attention_flops(spec, tokens, 0) \
        + 2 * spec.vocab_size * spec.hidden_size


def time_prefill(eng, tokens: int, repeats: int):
    import torch
    from safetyraise_lmengine_b200 import StepEntry
    gen = torch.Generator().manual_seed(1)
    times = []
    for i in range(repeats + 3):
        toks = torch.randint(0, eng.spec.vocab_size, (tokens,), generator=gen).tolist()
        s = eng.open_request()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        eng.step([StepEntry(s, toks, [tokens - 1])])
        b.record()
        torch.cuda.synchronize()
        eng.close_request(s)
        if i >= 3:                     # three runs warm up
            times.append(a.elapsed_time(b))
    return statistics.median(times)    # after the warm-ups the GPU sits at its power cap (sustained clocks)


def time_e2e(eng, batch: int, context: int, steps: int, warmup: int, ms_hint: float, min_seconds: float):
    """Decode through the Python entry point: requests are submitted as token ids, prefilled by the
    scheduler, and each timed step copies its token ids and batch layout from pinned host memory
    and reads the sampled tokens back to the host.  Blocks of `steps` steps by the wall clock with a
    synchronize on both sides; the median block."""
    import torch
    from safetyraise_lmengine_b200 import LLM, EngineConfig, SamplingParams
    from safetyraise_lmengine_b200.engine.scheduler import GenerationRequest
    cfg = EngineConfig(max_context=8192, max_active=batch, queue_capacity=batch, prefill_chunk=2048,
                       max_batch_tokens=eng.mctx.max_batch_tokens, page_size=PAGE_SIZE)
    llm = LLM(eng, cfg)
    llm.eos = set()
    nblocks = blocks_for(steps, warmup, ms_hint, min_seconds)
    gen = torch.Generator().manual_seed(2)
    for _ in range(batch):
        prompt = torch.randint(0, eng.spec.vocab_size, (context,), generator=gen).tolist()
        llm.submit(GenerationRequest(prompt, SamplingParams(temperature=0.0,
                                                            max_new_tokens=warmup + nblocks * steps + 8)))
    decoding = lambda: all(len(st.tokens) > st.usage.prompt_tokens for st in llm._live.values())
    while not decoding():
        llm.step()
    for _ in range(warmup):
        llm.step()
    seconds = []
    with ClockSampler() as clocks:
        for _ in range(nblocks):
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            for _ in range(steps):
                llm.step()
            torch.cuda.synchronize()
            seconds.append(time.perf_counter() - t0)
    time_e2e.clocks = clocks.summary()       # (of the last call: under a power cap the two arms may see other clocks)
    h2d = eng.last_h2d_bytes
    d2h = (8 + batch) * 4                                # the fault words and one token id per request
    for rid in list(llm._live):
        llm.cancel(rid)
    llm.step()
    assert eng.steps_failed == 0
    return batch * steps / statistics.median(seconds), h2d, d2h, nblocks


def kernel_table(eng, slots, context: int, top: int = 8):
    """Where the time of one eager decode step goes, kernel by kernel (events between the launches)."""
    import torch
    from safetyraise_lmengine_b200 import StepEntry
    from safetyraise_lmengine_b200.kernels import ops
    graphs, eng.use_graphs = eng.use_graphs, False
    try:
        for i in range(3):
            if i == 2:
                ops.begin_timing()
            eng.run(eng.prepare([StepEntry(s, [1 + i], [0]) for s in slots]))
        table = ops.end_timing()
    finally:
        eng.use_graphs = graphs
        rewind(eng, slots, context)
    total = sum(ms for _, ms in table.values()) or 1.0
    rows = sorted(table.items(), key=lambda kv: -kv[1][1])[:top]
    return {name: {"launches": n, "ms": round(ms, 3), "share": round(ms / total, 3)} for name, (n, ms) in rows}


def prefill_kernel_table(eng, tokens: int, top: int = 8):
    import torch
    from safetyraise_lmengine_b200 import StepEntry
    from safetyraise_lmengine_b200.kernels import ops
    s = eng.open_request()
    ops.begin_timing()
    eng.step([StepEntry(s, [7] * tokens, [tokens - 1])])
    table = ops.end_timing()
    eng.close_request(s)
    total = sum(ms for _, ms in table.values()) or 1.0
    rows = sorted(table.items(), key=lambda kv: -kv[1][1])[:top]
    return {name: {"launches": n, "ms": round(ms, 3), "share": round(ms / total, 3)} for name, (n, ms) in rows}


def config_record(shape: str, cfg: dict, layers: int, batch: int, context: int, workload: str) -> dict:
    return {"model": f"Qwen3-{shape.upper()} layer sizes", "layers": layers, "layers_of_config": cfg["num_hidden_layers"],
            "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
            "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
            "global_batch": batch, "seq_len": context, "benchmark_context": 4096, "page_size": PAGE_SIZE,
            "workload": workload, "parallelism": "single GPU",
            "l2": "not flushed: each step reads far more weight bytes than the 126 MB L2 holds"}


def run_decode(args, shape: str, pk) -> dict:
    import torch
    cfg = SHAPES[shape]
    B = args.batch or BATCH[shape]
    context = CONTEXT[shape]
    point_batches = [b for b in ((1, 64) if shape != "32b" else (1,)) if b != B]
    big = max([B] + point_batches)
    eng = build_engine(cfg, args.layers or cfg["num_hidden_layers"], max_requests=big,
                       tokens_in_cache=big * (context + MAX_GROWTH + 16) + PREFILL_TOKENS,
                       max_batch_tokens=PREFILL_TOKENS, graphs=not args.no_graphs)
    if args.only_prefill:
        return {"prefill_ms": time_prefill(eng, PREFILL_TOKENS, 5), "tokens": PREFILL_TOKENS}
    randomize_cache(eng)
    slots = fill_contexts(eng, B, context)
    with ClockSampler() as clocks:
        d = time_decode(eng, slots, context, args.steps, args.warmup, args.min_seconds)
    ms = d["ms_per_step"]
    nbytes = decode_bytes(eng, B, d["mean_context"])
    achieved = nbytes / (ms / 1000.0) / 1e9
    layers = len(eng.spec.run_order)
    out = {
        "metric": "decode_tokens_per_second", "value": round(B / (ms / 1000.0), 1), "unit": "tokens/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights N(0,0.02), uniform random token ids, random cache contents",
        "impl": "ours",
        "config": config_record(shape, cfg, layers, B, context, "decode"),
        "clocks": clocks.summary(),
        "gpu_launches": d["launches"],
        "timing": {"what": "median block of --steps whole steps (host and device half), CUDA events",
                   "blocks": d["blocks"], "timed_seconds": round(d["timed_seconds"], 2),
                   "device_half_ms": round(d["device_half_ms"], 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "bytes_per_step": nbytes,
                     "peak_source": pk["source"]},
    }
    if args.skip_extras:
        return out
    # the same step launched kernel by kernel (no CUDA graph), and where its time goes
    graphs, eng.use_graphs = eng.use_graphs, False
    eager = time_decode(eng, slots, context, min(args.steps, 20), 3, 0.0)
    eng.use_graphs = graphs
    out["timing"]["eager_ms"] = round(eager["ms_per_step"], 4)
    out["kernels"] = {"decode_step_eager": kernel_table(eng, slots, context)}
    for s in slots:
        eng.close_request(s)
    points = {}
    for b in point_batches:
        sl = fill_contexts(eng, b, context)
        p = time_decode(eng, sl, context, max(5, args.steps // 2), 3, 1.0)
        points[f"decode_b{b}"] = round(b / (p["ms_per_step"] / 1000.0), 1)
        frac = decode_bytes(eng, b, p["mean_context"]) / (p["ms_per_step"] / 1000.0) / 1e9 / pk["hbm_gbs"]
        points[f"decode_b{b}_hbm_frac"] = round(frac, 4)
        for s in sl:
            eng.close_request(s)
    pf_ms = time_prefill(eng, PREFILL_TOKENS, 5)
    flops = prefill_flops(eng.spec, PREFILL_TOKENS)
    out["prefill"] = {"value": round(PREFILL_TOKENS / (pf_ms / 1000.0), 1), "tokens": PREFILL_TOKENS,
                      "ms": round(pf_ms, 3),
                      "frac": round(flops / (pf_ms / 1000.0) / (pk["bf16_tflops"] * 1e12), 4),
                      "frac_of_sustained": round(flops / (pf_ms / 1000.0) / (pk["bf16_tflops_sustained"] * 1e12), 4),
                      "tflops": round(flops / (pf_ms / 1000.0) / 1e12, 1),
                      "regime": "sustained: median of 5 runs after 3 warm-ups, back to back"}
    out["kernels"]["prefill"] = prefill_kernel_table(eng, PREFILL_TOKENS)
    e2e, h2d, d2h, nb = time_e2e(eng, B, context, args.steps, args.warmup, ms, args.min_seconds)
    e2e_bytes = decode_bytes(eng, B, context + args.warmup + nb * args.steps // 2)
    out["e2e"] = {"value": round(e2e, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h,
                  "blocks": nb, "hbm_frac": round(e2e_bytes * e2e / B / 1e9 / pk["hbm_gbs"], 4),
                  "sm_mhz": time_e2e.clocks.get("sm_mhz"), "reasons": time_e2e.clocks.get("reasons")}
    for b in point_batches:
        v, _, _, nbp = time_e2e(eng, b, context, max(5, args.steps // 2), 3, 1000.0 * b / points[f"decode_b{b}"], 1.0)
        points[f"e2e_b{b}"] = round(v, 1)
    out["points"] = points
    return out


def run_mixed(args, shape: str, pk) -> dict:
    """32 requests, prompt lengths uniform in [128, 3072] from a seed, prefilled in portions of up to 512
    tokens beside the decoding requests, through the scheduler; every request generates --new-tokens."""
    import random

    import torch
    from safetyraise_lmengine_b200 import LLM, EngineConfig, SamplingParams
    from safetyraise_lmengine_b200.engine.scheduler import GenerationRequest
    cfg = SHAPES[shape]
    n_req, chunk, new = 32, 512, args.new_tokens
    rng = random.Random(0)
    lens = [rng.randint(128, 3072) for _ in range(n_req)]
    eng = build_engine(cfg, args.layers or cfg["num_hidden_layers"], max_requests=n_req,
                       tokens_in_cache=sum(lens) + n_req * (new + PAGE_SIZE), max_batch_tokens=chunk,
                       graphs=not args.no_graphs)
    spec = eng.spec
    ecfg = EngineConfig(max_context=4096, max_active=n_req, queue_capacity=n_req, prefill_chunk=chunk,
                        max_batch_tokens=chunk, page_size=PAGE_SIZE)
    gen = torch.Generator().manual_seed(3)
    prompts = [torch.randint(0, spec.vocab_size, (n,), generator=gen).tolist() for n in lens]

    def one_pass(timed: bool):
        llm = LLM(eng, ecfg)
        llm.eos = set()
        for p in prompts:
            llm.submit(GenerationRequest(p, SamplingParams(temperature=0.0, max_new_tokens=new)))
        steps = []
        torch.cuda.synchronize()
        t_all = time.perf_counter()
        while True:
            t0 = time.perf_counter()
            llm.last_step = None
            if not llm.step():
                break
            torch.cuda.synchronize()
            if llm.last_step is not None:
                steps.append((time.perf_counter() - t0, llm.last_step))
        return time.perf_counter() - t_all, steps, llm.metrics()

    from safetyraise_lmengine_b200.kernels import ops
    one_pass(False)                                   # warm-up: graphs recorded, buffers sized
    launches_before = ops.launches
    with ClockSampler() as clocks:
        seconds, steps, metrics = one_pass(True)
    launches = ops.launches - launches_before         # (a replayed graph counts the launches it holds)
    per_token = linear_flops_per_token(spec)
    weight_bytes = eng.model.weight_bytes() - spec.vocab_size * spec.hidden_size * 2
    kv_bytes_per_token = eng.cache.bytes_per_page() // eng.cache.page_size
    kinds = {"decode": [0.0, 0, 0.0], "portion": [0.0, 0, 0.0]}       # seconds, steps, work (bytes or flops)
    for sec, st in steps:
        counts, starts = st["counts"], st["starts"]
        if max(counts) == 1:
            k = kinds["decode"]
            k[2] += weight_bytes + sum(s + 1 for s in starts) * kv_bytes_per_token
        else:
            k = kinds["portion"]
            k[2] += sum(counts) * per_token + sum(attention_flops(spec, c, s) for c, s in zip(counts, starts)) \
                + 2.0 * len(counts) * spec.vocab_size * spec.hidden_size      # at most one logits row an entry
        k[0] += sec
        k[1] += 1
    total_tokens = sum(lens) + n_req * new
    dec, por = kinds["decode"], kinds["portion"]
    return {
        "metric": "mixed_tokens_per_second", "value": round(total_tokens / seconds, 1), "unit": "tokens/s",
        "n_gpus": 1, "steps": len(steps), "warmup": 1, "ms_per_step": round(1000.0 * seconds / len(steps), 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights N(0,0.02), prompts of uniform random token ids, lengths uniform in "
                "[128, 3072] from seed 0",
        "impl": "ours",
        "config": dict(config_record(shape, cfg, len(spec.run_order), n_req, 0, "mixed"), prefill_chunk=chunk,
                       new_tokens=new, prompt_tokens=sum(lens)),
        "clocks": clocks.summary(),
        "gpu_launches": launches,
        "generated_tokens_per_second": round(n_req * new / seconds, 1),
        "seconds": round(seconds, 3),
        "decode_steps": {"steps": dec[1], "mean_ms": round(1000.0 * dec[0] / max(dec[1], 1), 3),
                         "hbm_frac": round(dec[2] / max(dec[0], 1e-9) / 1e9 / pk["hbm_gbs"], 4)},
        "portion_steps": {"steps": por[1], "mean_ms": round(1000.0 * por[0] / max(por[1], 1), 3),
                          "tflops": round(por[2] / max(por[0], 1e-9) / 1e12, 1),
                          "frac": round(por[2] / max(por[0], 1e-9) / (pk["bf16_tflops"] * 1e12), 4),
                          "frac_of_sustained": round(por[2] / max(por[0], 1e-9) / (pk["bf16_tflops_sustained"] * 1e12), 4)},
        "scheduler": {k: int(v) for k, v in metrics.items()},
        "peak_source": pk["source"],
    }


# ---- Nekedra beside the Qwen3 decoder at equal layer sizes (--design nekedra) ---------------------------------
DESIGN_SIZES = {"2048": dict(width=2048, heads=16, kv_heads=4), "4096": dict(width=4096, heads=32, kv_heads=8)}
DESIGN_VOCAB = 32768
DESIGN_LAYERS = 4


def nekedra_config(size: dict, kinds) -> dict:
    """A Nekedra configuration whose layers have the sizes of a Qwen3 layer of the same width: heads of 128,
    a feed-forward of three widths; the latent of 512 with a rotated part of 64 per head."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    mixers = {
        "attention": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "v_mix": True},
        "latent_attention": {"heads": H, "dim": 128, "rot_dim": 64, "rot": {"base": 1e6, "dims": 64}, "kv_rank": 512,
                             "vdim": 128, "scale": 192 ** -0.5},
        "delta": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4},
    }
    return {"architecture": "Nekedra", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6},
            "layers": [{"type": k, "mixer": mixers[k], "mlp": {"kind": "dense", "ff": 3 * W}} for k in kinds]}


TONANEX_WINDOW = 1024
TONANEX_EXPERTS, TONANEX_TOP = 16, 4


def tonanex_config(size: dict, kinds) -> dict:
    """A Tonanex configuration whose layers have the sizes of a Qwen3 layer of the same width: heads of 128 for keys
    and values, a window of 1,024 tokens; a dense feed-forward of three widths, or 16 experts of half a width of which
    a token runs 4, plus a shared one of one width: three widths of feed-forward rows a token, as in the dense layer."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    mixer = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": TONANEX_WINDOW}}
    mlps = {"dense": {"kind": "dense", "ff": 3 * W},
            "moe": {"kind": "moe", "expert": {"ff": W // 2, "limit": 7.0},
                    "router": {"experts": TONANEX_EXPERTS, "top": TONANEX_TOP}, "shared": {"ff": W, "limit": 7.0}}}
    return {"architecture": "Tonanex", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": [{"type": "attention", "mixer": mixer, "mlp": mlps[k]} for k in kinds]}


PABALORN_WINDOW = 1024
PABALORN_EXPERTS, PABALORN_TOP = 16, 4


def pabalorn_config(size: dict, kinds) -> dict:
    """A Pabalorn configuration whose layers have the sizes of a Qwen3 layer of the same width: heads of 128 for keys
    and values with half of each head rotated, a window of 1,024 tokens and scores capped at 30; beside the attention
    of a 'parallel' layer a selective scan of two widths of channels with 16 states each; 16 experts of three quarters
    of a width of which a token runs 4: three widths of feed-forward rows a token, as in the dense layer."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    att = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": PABALORN_WINDOW},
           "rot": {"base": 10000.0, "dims": 64}}
    left = dict(att, rot={"base": 10000.0, "dims": 128,
                          "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}})
    right = {"inner": 2 * W, "state": 16, "dt_rank": W // 16, "conv": 4}
    mixers = {"attention": dict(att, softcap=30.0), "parallel": {"left": left, "right": right}}
    mlp = {"kind": "moe", "expert": {"ff": 3 * W // 4}, "router": {"experts": PABALORN_EXPERTS, "top": PABALORN_TOP}}
    return {"architecture": "Pabalorn", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6},
            "layers": [{"type": k, "mixer": mixers[k], "mlp": mlp} for k in kinds]}


DOVORAX_WINDOW = 1024


def dovorax_config(size: dict, kinds) -> dict:
    """A Dovorax configuration whose layers have the sizes of a Qwen3 layer of the same width: a latent attention with
    heads of 128 + 64, a latent of 512, a query latent of three quarters of a width and a window of 1,024 tokens; a
    'parallel' layer of attention with heads of 128 behind convolutions of 4 taps beside a matrix memory of half as
    many heads of 128 x 128; a gated linear recurrence of one width in blocks of 128 channels, 4 taps; the first
    layer's feed-forward dense (three widths), the others' 16 ungated experts of three quarters of a width in 4 groups
    of which 2 are kept, 4 a token, plus a shared one of one width and a half."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    scaling = {"factor": 16.0, "original": 4096, "fast": 24.0, "slow": 2.0}
    mixers = {
        "latent_attention": {"heads": H, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": 3 * W // 4,
                             "scale": 192 ** -0.5, "mask": {"size": DOVORAX_WINDOW},
                             "rot": {"base": 10000.0, "dims": 64, "scaling": scaling}},
        "parallel": {"left": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "conv": 4, "scale": 128 ** -0.5,
                              "rot": {"base": 10000.0, "dims": 64, "scaling": scaling}},
                     "right": {"heads": H // 2, "dim": 128, "vdim": 128, "gate_cap": 15.0},
                     "left_scale": 0.7, "right_scale": 0.7},
        "rglru": {"width": W, "blocks": W // 128, "conv": 4},
    }
    moe = {"kind": "moe", "expert": {"ff": 3 * W // 4}, "shared": {"ff": 3 * W // 2},
           "router": {"experts": 16, "top": 4, "groups": {"count": 4, "keep": 2}}}
    return {"architecture": "Dovorax", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6}, "postln_alpha": 2.0,
            "layers": [{"type": k, "mixer": mixers[k], "mlp": {"kind": "dense", "ff": 3 * W} if i == 0 else moe}
                       for i, k in enumerate(kinds)]}


LOKIZEN_WINDOW, LOKIZEN_KEPT = 1024, 16


def lokizen_config(size: dict, kinds) -> dict:
    """A Lokizen configuration whose layers have the sizes of a Qwen3 layer of the same width: attention with heads of 128
    for keys and values, a window of 1,024 tokens that keeps the first 16 and biases of distances up to 2,048; a
    retention of as many heads of 128 x 128, all of each head rotated; 16 ungated experts of three quarters of a width
    of which a token runs 4: three widths of feed-forward rows a token.  'loop' in the list: the layer behind it runs
    twice."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    mixers = {
        "attention": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "bias_max": 2048,
                      "mask": {"size": LOKIZEN_WINDOW, "keep_first": LOKIZEN_KEPT}},
        "retention": {"heads": H, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128},
                      "decay": [1.0 - 2.0 ** (-5.0 - 7.0 * h / H) for h in range(H)]},
    }
    mlp = {"kind": "moe", "expert": {"ff": 3 * W // 4}, "router": {"experts": 16, "top": 4, "scale": 1.5}}
    cfg = {"architecture": "Lokizen", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
           "layers": [{"type": k, "mixer": mixers[k], "mlp": mlp} for k in kinds if k != "loop"]}
    if "loop" in kinds:
        at = kinds.index("loop")
        cfg["loop"] = {"start": at, "stop": at + 1, "times": 2}
    return cfg


def mapovik_config(size: dict, kinds) -> dict:
    """A Mapovik configuration whose layers have the sizes of a Qwen3 layer of the same width: a delta rule of as many heads
    of 128 x 128 with half as many q / k heads, 4 taps and low-rank projections of the rank that generated weights get, 32; a
    'parallel' layer of attention with heads of 128, half of each rotated, beside a state space of two widths of channels in
    heads of 64 with 128 states, 4 taps; 16 gated experts of three quarters of a width of which a token's row of a table
    names 4, or ('... dense') a dense feed-forward of four and a half widths without a gate.  'loop' in the list: the layer
    behind it runs twice."""
    W, H, G = size["width"], size["heads"], size["kv_heads"]
    mixers = {
        "channel_delta": {"heads": H, "kv_heads": H // 2, "dim": 128, "vdim": 128, "conv": 4},
        "parallel": {"left": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                              "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0}}},
                     "right": {"heads": 2 * W // 64, "vdim": 64, "state": 128, "groups": 4, "norm_groups": 4, "conv": 4}},
    }
    moe = {"kind": "moe", "expert": {"ff": 3 * W // 4}, "router": {"experts": 16, "top": 4}}
    cfg = {"architecture": "Mapovik", "width": W, "vocab": DESIGN_VOCAB, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
           "logit_scale": 0.25,
           "layers": [{"type": k.removesuffix(" dense"), "mixer": mixers[k.removesuffix(" dense")],
                       "mlp": {"kind": "dense", "ff": 9 * W // 2} if k.endswith(" dense") else moe}
                      for k in kinds if k != "loop"]}
    if "loop" in kinds:
        at = kinds.index("loop")
        cfg["loop"] = {"start": at, "stop": at + 1, "times": 2}
    return cfg


def qwen3_config(size: dict) -> dict:
    return dict(BASE, num_hidden_layers=DESIGN_LAYERS, hidden_size=size["width"], num_attention_heads=size["heads"],
                num_key_value_heads=size["kv_heads"], intermediate_size=3 * size["width"], vocab_size=DESIGN_VOCAB)


def run_design(args) -> dict:
    """Prefill (2,048 tokens, one request) and decode (batch 8 behind 2,048 tokens) of four-layer models with
    random weights: the Qwen3 decoder, and Nekedra stacks of each mixer alone and of all three, at equal
    widths, heads and feed-forward sizes.  Times of whole steps through the step function, CUDA events,
    three warm-ups; beside each the kernels that take the most time of an eager step."""
    import torch
    batch, context = 8, CONTEXT["8b"]
    stacks = {"qwen3": None, "nekedra attention": ["attention"] * DESIGN_LAYERS,
              "nekedra latent": ["latent_attention"] * DESIGN_LAYERS, "nekedra delta": ["delta"] * DESIGN_LAYERS,
              "nekedra mixed": ["latent_attention", "delta", "attention", "delta"]}
    make = nekedra_config
    if args.design == "tonanex":
        stacks = {"qwen3": None, "tonanex dense": ["dense"] * DESIGN_LAYERS, "tonanex experts": ["moe"] * DESIGN_LAYERS}
        make = tonanex_config
    if args.design == "pabalorn":
        stacks = {"qwen3": None, "tonanex experts": ["moe"] * DESIGN_LAYERS,
                  "pabalorn attention": ["attention"] * DESIGN_LAYERS, "pabalorn parallel": ["parallel"] * DESIGN_LAYERS,
                  "pabalorn mixed": ["attention", "parallel"] * (DESIGN_LAYERS // 2)}
        make = lambda size, kinds: (tonanex_config if kinds[0] == "moe" else pabalorn_config)(size, kinds)
    if args.design == "dovorax":
        stacks = {"qwen3": None, "nekedra latent": ["latent_attention"] * DESIGN_LAYERS, "nekedra delta": ["delta"] * DESIGN_LAYERS,
                  "tonanex experts": ["moe"] * DESIGN_LAYERS,
                  "dovorax latent": ["latent_attention"] * DESIGN_LAYERS, "dovorax parallel": ["parallel"] * DESIGN_LAYERS,
                  "dovorax recurrence": ["rglru"] * DESIGN_LAYERS,
                  "dovorax mixed": ["latent_attention", "parallel", "rglru", "latent_attention"]}
        make = lambda size, kinds: (tonanex_config if kinds[0] == "moe" else nekedra_config if kinds[0] == "delta" else None)(size, kinds)
    if args.design == "lokizen":
        stacks = {"qwen3": None, "tonanex experts": ["moe"] * DESIGN_LAYERS, "nekedra delta": ["delta"] * DESIGN_LAYERS,
                  "lokizen attention": ["attention"] * DESIGN_LAYERS, "lokizen retention": ["retention"] * DESIGN_LAYERS,
                  "lokizen looped": ["retention", "loop", "attention", "retention"]}
        make = tonanex_config
    if args.design == "mapovik":
        stacks = {"qwen3": None, "nekedra delta": ["delta"] * DESIGN_LAYERS, "tonanex experts": ["moe"] * DESIGN_LAYERS,
                  "pabalorn parallel": ["parallel"] * DESIGN_LAYERS,
                  "mapovik delta": ["channel_delta"] * DESIGN_LAYERS, "mapovik parallel": ["parallel"] * DESIGN_LAYERS,
                  "mapovik looped": ["channel_delta dense", "loop", "parallel", "channel_delta"]}
        make = lambda size, kinds: (tonanex_config if kinds[0] == "moe" else pabalorn_config)(size, kinds)
    out = {"metric": args.design + "_beside_qwen3", "layers": DESIGN_LAYERS, "prefill_tokens": PREFILL_TOKENS,
           "decode_batch": batch, "decode_context": context, "dtype": "bf16", "data": "synthetic", "sizes": {}}
    sizes = [args.design_size] if args.design_size else sorted(DESIGN_SIZES)
    for name in sizes:
        size, rows = DESIGN_SIZES[name], {}
        for label, kinds in stacks.items():
            if args.design_stack and not label.startswith(args.design_stack):
                continue
            if label.startswith("dovorax"):
                cfg = dovorax_config(size, kinds)
            elif label.startswith("lokizen"):
                cfg = lokizen_config(size, kinds)
            elif label.startswith("mapovik"):
                cfg = mapovik_config(size, kinds)
            elif label.startswith("nekedra"):
                cfg = nekedra_config(size, kinds)
            else:
                cfg = qwen3_config(size) if kinds is None else make(size, kinds)
            eng = build_engine(cfg, DESIGN_LAYERS, batch + 1, batch * (context + MAX_GROWTH) + PREFILL_TOKENS,
                               PREFILL_TOKENS)
            randomize_cache(eng)
            prefill_ms = time_prefill(eng, PREFILL_TOKENS, 3)
            ptable = prefill_kernel_table(eng, PREFILL_TOKENS, top=args.design_kernels)
            slots = fill_contexts(eng, batch, context)
            d = time_decode(eng, slots, context, args.steps, args.warmup, 0.5)
            dtable = kernel_table(eng, slots, context, top=args.design_kernels)
            rows[label] = {"prefill_ms": round(prefill_ms, 3),
                           "prefill_tok_s": round(PREFILL_TOKENS / prefill_ms * 1000.0, 1),
                           "decode_ms_per_step": round(d["ms_per_step"], 4),
                           "decode_tok_s": round(batch / d["ms_per_step"] * 1000.0, 1),
                           "decode_launches_per_step": d["launches"] // max(args.steps, 1),
                           "weight_bytes": eng.model.weight_bytes(),
                           "prefill_kernels": ptable, "decode_kernels": dtable}
            del eng, slots
            torch.cuda.empty_cache()
        out["sizes"][name] = rows
    return out


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=100)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--shape", default="8b", choices=sorted(SHAPES))
    ap.add_argument("--workload", default=None, choices=["decode", "mixed"],
                    help="decode (default; with prefill and the batch points) or mixed (default of --shape 14b)")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration has")
    ap.add_argument("--batch", type=int, default=0, help="decode batch (default 8; 64 for --shape 32b)")
    ap.add_argument("--new-tokens", type=int, default=128, help="mixed workload: tokens every request generates")
    ap.add_argument("--skip-extras", action="store_true", help="only the default decode measurement")
    ap.add_argument("--no-graphs", action="store_true", help="launch every kernel from the host (for profilers)")
    ap.add_argument("--only-prefill", action="store_true", help="run just the 2,048-token prefill (for profilers)")
    ap.add_argument("--streaming-kernel", action="store_true",
                    help="steps of up to 8 tokens on the weight-streaming mma.sync kernel instead of the tensor-core one")
    ap.add_argument("--design", default=None, choices=["nekedra", "tonanex", "pabalorn", "dovorax", "lokizen", "mapovik"],
                    help="instead of the default workload: prefill and decode of that design's stacks beside the Qwen3 decoder "
                         "at equal layer sizes")
    ap.add_argument("--design-stack", default=None, help="only the stacks of --design whose name begins so")
    ap.add_argument("--design-kernels", type=int, default=6, help="how many kernels of every step --design lists")
    ap.add_argument("--design-size", default=None, choices=sorted(DESIGN_SIZES), help="one width of --design")
    ap.add_argument("--min-seconds", type=float, default=MIN_TIMED_SECONDS,
                    help="repeat the block of --steps steps until this much is timed (0: one block, for profilers)")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not offered")
        return 2
    args.warmup = max(args.warmup, 3)
    workload = args.workload or ("mixed" if args.shape == "14b" else "decode")
    if args.streaming_kernel:
        from safetyraise_lmengine_b200.kernels import ops
        ops.skinny_max_tokens = 8
    if args.design:
        if args.steps == 100:
            args.steps = 20
        print(json.dumps(run_design(args)))
        return 0
    pk = peaks()
    out = run_mixed(args, args.shape, pk) if workload == "mixed" else run_decode(args, args.shape, pk)
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
