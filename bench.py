#!/usr/bin/env python3
"""Decode and prefill throughput of the engine on one GPU, as one JSON line.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

Default run: the layer sizes of Llama-3.2-1B with random bfloat16 weights, a batch of 8
sequences with 2,048-token prompts in a 4,096-token context; a "step" is one decode
step of the whole batch.  ``value`` is decoded tokens a second with the step timed on the
device (CUDA events on the engine's stream around K decode steps); ``e2e`` is the same through the Python entry
point (``Model.generate``), host token ids in and sampled ids out at every step.  The line
also carries the prefill of 2,048 tokens, the decode step's bytes against the memory
bandwidth, and decode at batch 1 and 64.  The decode step reads about 3 GB (weights and
cache), far more than the 126 MB L2, so no flush is needed between steps.
Only one GPU is supported: for --gpus N > 1 it says so and exits with 2."""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

LLAMA_1B = dict(model_type="llama", num_hidden_layers=16, hidden_size=2048, num_attention_heads=32,
                num_key_value_heads=8, head_dim=64, intermediate_size=8192, vocab_size=128256,
                rope_theta=500000.0,
                rope_scaling=dict(rope_type="llama3", factor=32.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                  original_max_position_embeddings=8192),
                rms_norm_eps=1e-5, tie_word_embeddings=True, max_position_embeddings=131072,
                hidden_act="silu")
LLAMA_3B = dict(LLAMA_1B, num_hidden_layers=28, hidden_size=3072, num_attention_heads=24, num_key_value_heads=8,
                head_dim=128, intermediate_size=8192)
LLAMA_8B = dict(LLAMA_1B, num_hidden_layers=32, hidden_size=4096, num_attention_heads=32, num_key_value_heads=8,
                head_dim=128, intermediate_size=14336, tie_word_embeddings=False,
                rope_scaling=dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                  original_max_position_embeddings=8192))
CONTEXT = 4096
PROMPT = 2048
FALLBACK_PEAKS = dict(hbm_gbs=6650.0, bf16_tflops=1590.0)


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        with open(path) as f:
            p = json.load(f)
        return dict(hbm_gbs=float(p["hbm_gbs"]), bf16_tflops=float(p["bf16_tflops"]), source="measured")
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([x.strip() for x in line.split(",")])

    def stop(self):
        if self.proc is None:
            return dict(sm_mhz=None, sm_max_mhz=None, reasons=["nvidia-smi unavailable"])
        self.proc.terminate()
        self.thread.join(timeout=2)
        sm = [float(r[0]) for r in self.rows if len(r) >= 6 and r[0].replace(".", "").isdigit()]
        mx = [float(r[1]) for r in self.rows if len(r) >= 6 and r[1].replace(".", "").isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({names[i] for r in self.rows if len(r) >= 6 for i in range(4) if r[2 + i] == "Active"})
        # "under load": a run also spends time where the GPU idles at a few hundred MHz (a model file
        # being written, a process starting); those samples say nothing about the timed kernels
        busy = [x for x in sm if x >= 0.5 * max(sm)] if sm else []
        return dict(sm_mhz=statistics.median(busy) if busy else None, sm_max_mhz=max(mx) if mx else None,
                    reasons=reasons, samples=len(sm), samples_under_load=len(busy))


def model_numbers(c):
    """Bytes a decode step has to read per weight pass and per cached token; prefill flops."""
    H, L, I, V = c["hidden_size"], c["num_hidden_layers"], c["intermediate_size"], c["vocab_size"]
    nH, nKV, d = c["num_attention_heads"], c["num_key_value_heads"], c["head_dim"]
    per_layer = H * (nH + 2 * nKV) * d + nH * d * H + 3 * H * I + 2 * H
    weight_bytes = 2 * (L * per_layer + V * H + H)          # every weight used once, the output matrix included
    kv_bytes_per_token = 2 * L * nKV * d * 2

    def prefill_flops(T, rows=1):
        # what the step has to compute: the last layer's feed-forward and the output matrix only for
        # the rows whose logits are wanted (the engine does no more, so no more is counted)
        lin = 2 * T * L * (H * (nH + 2 * nKV) * d + nH * d * H) + 2 * (T * (L - 1) + rows) * 3 * H * I
        att = L * 4 * nH * d * T * (T + 1) // 2            # q k^T and p v over the causal half
        return lin + att + 2 * rows * V * H
    return weight_bytes, kv_bytes_per_token, prefill_flops


LAST_STEP_TIMES = []          # milliseconds of each timed step of the last decode_rate call


def products_alone(cfg, tokens, pk):
    """The step's dominant kernel by itself: the tcgen05 products of a whole step (every layer's four,
    each layer with weights of its own so that none is met in L2, then the output matrix) launched one
    behind the other as in the step (one CUDA graph), without the attention and the norms between them: bytes of weights
    over time against the measured bandwidth.  What the step loses beyond this is the other kernels
    and the hand-overs to and from them."""
    import torch
    from libllm_b200.csrc import ops
    H, I, V, L = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"], cfg["num_hidden_layers"]
    nH, nKV, d = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    bf = torch.bfloat16
    shapes = [((nH + 2 * nKV) * d, H, False), (H, nH * d, False), (2 * I, H, True), (H, I, False)]
    jobs, nbytes = [], 0.0
    for layer in range(L + 1):
        for n, k, sw in (shapes if layer < L else [(V, H, False)]):
            x = torch.randn(tokens, k, device="cuda").to(bf)
            w = torch.empty(n, k, device="cuda", dtype=bf).normal_(0.0, 0.02)
            n_out = n // 2 if sw else n
            parts = 1 if sw or n == V else ops.gemm_tc_suggest_parts(tokens, n, k)
            out = torch.empty((tokens, n_out) if parts == 1 else (parts, tokens, n_out), dtype=bf if sw else torch.float32, device="cuda")
            jobs.append((x, w, out, sw))
            nbytes += 2.0 * n * k
    def run():
        for x, w, out, sw in jobs:
            ops.gemm_tc(x, w, out, swiglu=sw)
    side = torch.cuda.Stream()
    with torch.cuda.stream(side):
        run()                                    # outside capture once: attributes, tensor maps
        side.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=side):
            run()
        times = []
        for rep in range(6):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record(side)
            graph.replay()
            b.record(side)
            b.synchronize()
            if rep >= 2:
                times.append(a.elapsed_time(b) * 1e3)
    us = statistics.median(times)
    gbs = nbytes / (us * 1e-6) / 1e9
    return {"kernel": "gemm_tc_kernel: the step's products one behind the other, nothing between them",
            "launches": len(jobs), "us_per_step": round(us, 1), "gb_s": round(gbs, 1), "frac": round(gbs / pk["hbm_gbs"], 4)}


def decode_rate(model, batch, steps, warmup, vocab, seed=0):
    """Decoded tokens a second at ``batch`` with the steps timed on the device: CUDA events on the
    engine's stream around ``steps`` decode steps that are queued one behind the other (each takes
    its tokens from the one before on the device, so nothing waits for the host; the host queues a
    step in a small part of the time the device takes to run one).  Also returns the kernel
    launches of one step, counted by the host library while the step's graph was made."""
    import torch
    from libllm_b200 import _lib
    from libllm_b200.engine import GREEDY, StepItem
    eng = model.engine
    stream = torch.cuda.ExternalStream(eng.stream)
    g = torch.Generator().manual_seed(seed)
    slots = [eng.open_sequence() for _ in range(batch)]
    try:
        prompts = torch.randint(0, vocab, (batch, PROMPT), generator=g).tolist()
        # prompts in one step (the engine cuts it into launches of max_step_tokens)
        eng.step_tokens([StepItem(s, p, [PROMPT - 1]) for s, p in zip(slots, prompts)], GREEDY).result()
        fed = [StepItem(s, [0], [0], fed_row=i) for i, s in enumerate(slots)]
        n0 = _lib.lib().llm_kernel_launches()
        eng.step_tokens(fed, GREEDY).result()          # a shape's first step runs once and is captured once
        launches = (_lib.lib().llm_kernel_launches() - n0) // 2
        for _ in range(max(warmup - 1, 2)):
            eng.step_tokens(fed, GREEDY).result()
        marks = [torch.cuda.Event(enable_timing=True) for _ in range(steps + 1)]
        eng.synchronize()
        marks[0].record(stream)
        pending = []
        for i in range(steps):
            pending.append(eng.step_tokens(fed, GREEDY))
            marks[i + 1].record(stream)
        for p in pending:
            p.result()
        eng.synchronize()
        ms = marks[0].elapsed_time(marks[steps]) / steps          # the K steps as one stretch: the record's figure
        LAST_STEP_TIMES[:] = [marks[i].elapsed_time(marks[i + 1]) for i in range(steps)]
        ctx_len = eng.sequence_length(slots[0])
        return batch * 1000.0 / ms, ms, ctx_len, launches
    finally:
        for s in slots:
            eng.close_sequence(s)


def e2e_rate(model, batch, steps, warmup, vocab, seed=1):
    """Decoded tokens a second through Model.generate, the call a user makes: token ids go in as
    Python lists and come out as Python lists.  Every step copies its descriptor (positions, page
    tables, token sources) from pinned host memory to the device and reads the sampled ids back;
    the clock is the host's, stamped when a step's tokens have arrived."""
    import torch
    g = torch.Generator().manual_seed(seed)
    prompts = torch.randint(0, vocab, (batch, PROMPT), generator=g).tolist()
    stamps = []

    def on_token(i, tok):
        if i == 0:
            stamps.append(time.perf_counter())

    model.generate(prompts, max_new_tokens=warmup + steps + 1, temperature=0.0, top_k=1, top_p=1.0, seed=0,
                   stop_token_ids=[], max_batch=batch, on_token=on_token)
    # stamps[0] follows the prompt step; steps warmup+1 .. warmup+steps are timed
    t = stamps[warmup + steps] - stamps[warmup]
    info = model.engine.info()
    return batch * steps / t, info["last_step_h2d_bytes"], info["last_step_d2h_bytes"]


def prefill_rate(model, vocab, flops_fn, peak_tflops, reps=3):
    import torch
    from libllm_b200.engine import StepItem
    eng = model.engine
    stream = torch.cuda.ExternalStream(eng.stream)
    g = torch.Generator().manual_seed(7)
    prompt = torch.randint(0, vocab, (PROMPT,), generator=g).tolist()
    times = []
    for r in range(reps + 2):
        s = eng.open_sequence()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        eng.synchronize()
        a.record(stream)
        eng.step([StepItem(s, prompt, [PROMPT - 1])])      # returns when the wanted row's logits are in host memory
        b.record(stream)
        eng.synchronize()
        eng.close_sequence(s)
        if r >= 2:
            times.append(a.elapsed_time(b))
    ms = statistics.median(times)
    flops = flops_fn(PROMPT)
    return dict(value=PROMPT * 1000.0 / ms, tokens=PROMPT, ms=ms, frac=flops / (ms * 1e-3) / (peak_tflops * 1e12))


def run_workload(args):
    """The two larger workloads the benchmark description names, through Model.generate (host token ids in
    and out): Llama-3.2-3B sizes with 16 prompts of lengths uniform in [128, 2048] and 256 decoded tokens
    each; Llama-3.1-8B sizes with 32 prompts of 4,096 tokens and 512 decoded tokens each.  One JSON line:
    time to the first tokens (all prompts in one step), decoded tokens a second after it, and the bytes
    the decode steps had to read against the memory bandwidth."""
    import torch
    from libllm_b200 import Model
    if args.workload == "3b":
        cfg, n_new = dict(LLAMA_3B), 256
        g = torch.Generator().manual_seed(11)
        lens = torch.randint(128, 2049, (16,), generator=g).tolist()
        context = 2048 + n_new
    else:
        cfg, n_new = dict(LLAMA_8B), 512
        lens = [4096] * 32
        context = 8192
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    g = torch.Generator().manual_seed(12)
    prompts = [torch.randint(0, cfg["vocab_size"], (n,), generator=g).tolist() for n in lens]
    pages = sum((n + n_new + 63) // 64 for n in lens)
    model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=pages * 64, max_seq_len=context)
    stamps = []

    def on_token(i, tok):
        if i == 0:
            stamps.append(time.perf_counter())

    model.generate(prompts[:2], max_new_tokens=4, temperature=0.0, stop_token_ids=[])        # kernels loaded, graphs not
    t0 = time.perf_counter()
    out = model.generate(prompts, max_new_tokens=n_new, temperature=0.0, stop_token_ids=[], max_batch=len(prompts),
                         on_token=on_token)
    t1 = time.perf_counter()
    assert all(len(o) == n_new for o in out)
    wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
    pk = peaks()
    ttft = stamps[0] - t0
    decode_s = t1 - stamps[0]
    steps = n_new - 1
    mean_ctx = sum(lens) / len(lens) + n_new / 2
    step_bytes = wbytes + len(lens) * mean_ctx * kv_per_tok
    prefill_flops = sum(flops_fn(n) for n in lens)
    print(json.dumps({
        "workload": args.workload, "impl": "ours", "dtype": "bf16", "data": "synthetic",
        "config": {"layers": cfg["num_hidden_layers"], "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "batch": len(lens),
                   "prompt_tokens": sum(lens), "new_tokens_each": n_new},
        "prefill": {"tokens": sum(lens), "ms": round(ttft * 1e3, 2), "tok_s": round(sum(lens) / ttft, 1),
                    "frac": round(prefill_flops / ttft / (pk["bf16_tflops"] * 1e12), 4)},
        "decode": {"tok_s": round(len(lens) * steps / decode_s, 1), "ms_per_step": round(decode_s / steps * 1e3, 3),
                   "hbm_frac": round(step_bytes / (decode_s / steps) / 1e9 / pk["hbm_gbs"], 4)},
        "total_s": round(t1 - t0, 3)}))
    return 0


# ---------------------------------------------------------------- Sinezen beside Llama at equal sizes
def sinezen_config(hidden, runs, heads, kv, dim, ff, vocab, mask, moe=None):
    """A Sinezen model of `runs` layer runs: two layers before a loop of two layers that repeats as
    often as the runs ask for.  `moe` = (experts, top, expert ff, shared ff) puts a routed feed-forward
    into every second layer."""
    mixer = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, mask=dict(size=mask),
                 rot=dict(base=500000.0, dims=dim))
    dense = dict(kind="dense", ff=ff)
    routed = dense if moe is None else dict(kind="moe", router=dict(experts=moe[0], top=moe[1]), expert=dict(ff=moe[2]),
                                            shared=dict(ff=moe[3]))
    layer = lambda mlp: dict(type="attention", mixer=mixer, mlp=mlp)
    times = max(1, (runs - 2) // 2)
    return dict(architecture="Sinezen", vocab=vocab, width=hidden, norm=dict(eps=1e-5),
                layers=[layer(dense), layer(routed), layer(dense), layer(routed)], loop=dict(start=2, stop=4, times=times))


def sinezen_numbers(c, batch):
    """(bytes a decode step reads at `batch` apart from the cache, cache bytes per visible token,
    prefill flops of T tokens with one wanted row) for a Sinezen configuration."""
    H, V = c["width"], c["vocab"]
    loop = c["loop"]
    runs = list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + \
        list(range(loop["stop"], len(c["layers"])))

    def layer_mats(L, tokens):
        """(matrix values every token uses, matrix values the step reads) of one layer"""
        m, f = L["mixer"], L["mlp"]
        att = H * (m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"]) + m["heads"]) + m["heads"] * m["vdim"] * H
        if f["kind"] == "dense":
            return att + 3 * H * f["ff"], att + 3 * H * f["ff"]
        E, top, eff, sff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], f["shared"]["ff"]
        used = att + H * E + 2 * H * (top * eff + sff)
        return used, att + H * E + 2 * H * (min(E, tokens * top) * eff + sff)

    # a layer that runs twice is read twice: the runs between its two uses read more than L2 holds
    weight_bytes = 2 * (sum(layer_mats(c["layers"][i], batch)[1] for i in runs) + 2 * V * H + loop["times"] * 2 * H * H)
    kv_per_token = sum(2 * c["layers"][i]["mixer"]["kv_heads"] * (c["layers"][i]["mixer"]["dim"] + c["layers"][i]["mixer"]["vdim"]) for i in runs)

    def prefill_flops(T):
        lin = 2 * T * sum(layer_mats(c["layers"][i], T)[0] for i in runs) + loop["times"] * 2 * T * 2 * H * H
        att = 0
        for i in runs:
            m = c["layers"][i]["mixer"]
            B = m["mask"]["size"]
            full, rest = divmod(T, B)
            seen = full * B * (B + 1) // 2 + rest * (rest + 1) // 2
            att += 2 * m["heads"] * (m["dim"] + m["vdim"]) * seen
        return lin + att + 2 * V * H
    return weight_bytes, kv_per_token, prefill_flops


COMPARE_SIZES = {
    # name: (hidden, layer runs, heads, kv heads, head size, feed-forward, vocabulary, mask, routed)
    "2k": (2048, 8, 32, 8, 64, 8192, 32000, 1024, None),
    "4k": (4096, 4, 32, 8, 128, 14336, 32000, 2048, None),
    "2k-routed": (2048, 8, 32, 8, 64, 4096, 32000, 1024, (32, 4, 1024, 2048)),
}


# ---------------------------------------------------------------- Sesuzen beside Llama at equal sizes
def sesuzen_config(hidden, runs, heads, kv, dim, ff, vocab, window, keep, moe=None, taps=4, rank=64):
    """A Sesuzen model of `runs` layer runs: a delta-rule layer and an attention layer (a window of `window`
    positions that keeps the first `keep`) in a loop that repeats as often as the runs ask for.  `moe` =
    (experts, top, expert ff) puts a routed feed-forward into the attention layers."""
    attention = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, mask=dict(size=window, keep_first=keep))
    delta = dict(heads=hidden // dim, dim=dim, rank=rank)
    dense = dict(kind="dense", ff=ff)
    routed = dense if moe is None else dict(kind="moe", router=dict(experts=moe[0], top=moe[1]), expert=dict(ff=moe[2]))
    return dict(architecture="Sesuzen", vocab=vocab, width=hidden, max_positions=CONTEXT, norm=dict(eps=1e-5), canon=dict(taps=taps),
                logit_softcap=30.0, layers=[dict(type="general_delta", mixer=delta, mlp=dense), dict(type="attention", mixer=attention, mlp=routed)],
                loop=dict(start=0, stop=2, times=max(1, runs // 2)))


def sesuzen_numbers(c, batch):
    """(bytes a decode step reads at `batch` apart from the cache, cache bytes per visible token, bytes of recurrent
    state a step reads and writes per sequence, prefill flops of T tokens with one wanted row)."""
    H, V = c["width"], c["vocab"]
    loop = c["loop"]
    runs = list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], len(c["layers"])))

    def layer_mats(L, tokens):
        """(matrix values every token uses, matrix values the step reads) of one layer"""
        m, f = L["mixer"], L["mlp"]
        if L["type"] == "attention":
            mix = H * (m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"]) + m["heads"] * m["vdim"]) + m["heads"] * m["vdim"] * H
        else:
            W = m["heads"] * m["dim"]
            mix = 6 * H * W + m["rank"] * (H + 2 * W)             # r, k, v, g, a, o; the low-rank pair (the second in 32-bit)
        if f["kind"] == "dense":
            return mix + 2 * H * f["ff"], mix + 2 * H * f["ff"]
        E, top, eff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
        return mix + H * E + 3 * H * top * eff, mix + H * E + 3 * H * min(E, tokens * top) * eff

    weight_bytes = 2 * (sum(layer_mats(c["layers"][i], batch)[1] for i in runs) + V * H)
    att = [c["layers"][i]["mixer"] for i in runs if c["layers"][i]["type"] == "attention"]
    dl = [c["layers"][i]["mixer"] for i in runs if c["layers"][i]["type"] != "attention"]
    kv_per_token = sum(2 * m["kv_heads"] * (m["dim"] + m["vdim"]) for m in att)
    state_bytes = sum(2 * 4 * m["heads"] * m["dim"] * m["dim"] for m in dl)      # read and written, 32-bit

    def prefill_flops(T):
        lin = 2 * T * sum(layer_mats(c["layers"][i], T)[0] for i in runs)
        a = 0
        for m in att:
            w, k = m["mask"]["size"], m["mask"]["keep_first"]
            seen = sum(min(i + 1, w) + max(0, min(k, i + 1 - w)) for i in range(T))
            a += 2 * m["heads"] * (m["dim"] + m["vdim"]) * seen
        rec = sum(10 * m["heads"] * m["dim"] * m["dim"] * T for m in dl)       # decay, removal, outer product, read-out per column
        return lin + a + rec + 2 * V * H
    return weight_bytes, kv_per_token, state_bytes, prefill_flops


SESUZEN_SIZES = {
    # name: (hidden, layer runs, heads, kv heads, head size, feed-forward, vocabulary, window, kept first, routed)
    "2k": (2048, 8, 32, 8, 64, 8192, 32000, 1024, 4, None),
    "4k": (4096, 4, 32, 8, 128, 14336, 32000, 1024, 4, None),
    "2k-routed": (2048, 8, 32, 8, 64, 8192, 32000, 1024, 4, (32, 4, 2048)),
}


def run_compare_sesuzen(args):
    """Prefill and decode of Sesuzen beside Llama, both with random weights, at equal hidden size, layer runs, heads,
    head size and vocabulary; the feed-forward has two matrices of the width Llama's three have (with experts: the
    chosen ones' three): one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    names = [n for n in SESUZEN_SIZES if not args.sizes or n in args.sizes.split(",")]
    for name in names:
        hidden, runs, heads, kv, dim, ff, vocab, window, keep, routed = SESUZEN_SIZES[name]
        llama = dict(LLAMA_1B, num_hidden_layers=runs, hidden_size=hidden, num_attention_heads=heads, num_key_value_heads=kv,
                     head_dim=dim, intermediate_size=ff, vocab_size=vocab, tie_word_embeddings=False, rope_scaling=None)
        zen = sesuzen_config(hidden, runs, heads, kv, dim, ff, vocab, window, keep, routed)
        only = getattr(args, "model", None)
        for label, cfg in (("llama", llama), ("sesuzen", zen)):
            if only and only != label:
                continue
            state_bytes = 0
            if label == "llama":
                wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
                flops = flops_fn(PROMPT)
            else:
                wbytes, kv_per_tok, state_bytes, zen_flops = sesuzen_numbers(cfg, args.batch)
                flops = zen_flops(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            seen = ctx_len if label == "llama" else min(ctx_len, window + keep)
            step_bytes = wbytes + args.batch * (seen * kv_per_tok + state_bytes)
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "layer_runs": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "window": window if label == "sesuzen" else None,
                                         "kept_first": keep if label == "sesuzen" else None, "routed": routed if label == "sesuzen" else None},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": round(step_bytes / 1e9, 3),
                                         "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


# ---------------------------------------------------------------- Sobezen beside Llama at equal sizes
def sobezen_config(hidden, runs, heads, kv, dim, ff, vocab, kv_rank=512, taps=4, limit=7.0):
    """A Sobezen model of `runs` layers in the order delta rule, attention (values are the keys), latent attention with
    rows of its own, latent attention that reads the rows of the layer before it; every layer has the dense gated
    feed-forward.  The latent layers' heads have `dim` unrotated and dim / 2 rotated channels and a query latent of
    3 / 8 of the width."""
    rot = dict(dims=dim, base=1e4)
    rot_l = dict(dims=dim // 2, base=1e4, scaling=dict(factor=4.0, original=2048, fast=16.0, slow=2.0))
    mlp = dict(kind="dense", ff=ff, limit=limit)
    layers = []
    for i in range(runs):
        k = i % 4
        if k == 0:
            L = dict(type="channel_delta", mixer=dict(heads=hidden // dim, kv_heads=max(1, hidden // dim // 4), dim=dim, vdim=dim, conv=taps))
        elif k == 1:
            L = dict(type="attention", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, rot=rot))
        else:
            m = dict(heads=heads, dim=dim, rot_dim=dim // 2, vdim=dim, kv_rank=kv_rank, q_rank=hidden * 3 // 8,
                     scale=(dim + dim // 2) ** -0.5, rot=rot_l)
            if k == 3:
                m["kv_from"] = i - 1
            L = dict(type="latent_attention", mixer=m)
        layers.append(dict(mlp=mlp, **L))
    return dict(architecture="Sobezen", vocab=vocab, width=hidden, norm=dict(eps=1e-5), embedding=dict(scale=1.0), logit_scale=1.0,
                layers=layers)


SOBEZEN_FREE_RANK = 16        # the size Model.from_random gives the low-rank inputs' inner side


def sobezen_numbers(c):
    """(bytes a decode step reads apart from the cache, cache bytes per visible token, bytes of recurrent state a step
    reads and writes per sequence, prefill flops of T tokens with one wanted row)."""
    H, V = c["width"], c["vocab"]
    mats, kv_per_token, state_bytes, att_flops_per_key, rec_flops_per_token = 0, 0, 0, 0, 0
    for L in c["layers"]:
        m = L["mixer"]
        if L["type"] == "attention":
            mats += H * (m["heads"] + m["kv_heads"]) * m["dim"] + m["heads"] * m["dim"] * H
            kv_per_token += 2 * 2 * m["kv_heads"] * m["dim"]                                  # rotated keys and the keys as values
            att_flops_per_key += 2 * m["heads"] * 2 * m["dim"]
        elif L["type"] == "latent_attention":
            row = m["kv_rank"] + m["rot_dim"]
            mats += H * m["q_rank"] + m["q_rank"] * m["heads"] * (m["dim"] + m["rot_dim"]) + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"]
            mats += m["heads"] * m["vdim"] * H + (0 if "kv_from" in m else H * row)
            kv_per_token += 2 * row                                                           # a borrower reads the rows again
            att_flops_per_key += 2 * m["heads"] * (row + m["kv_rank"])
        else:
            qk, k, v, r = m["kv_heads"] * m["dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"], SOBEZEN_FREE_RANK
            mats += H * (2 * qk + v + m["heads"] + 2 * r) + v * H + 2 * r * (k + v)             # the second low-rank sides in 32-bit
            state_bytes += 2 * 4 * m["heads"] * m["dim"] * m["vdim"]
            rec_flops_per_token += 8 * m["heads"] * m["dim"] * m["vdim"]                       # decay, prediction, write, read-out
        if L["mlp"]:
            mats += 3 * H * L["mlp"]["ff"]
    weight_bytes = 2 * (mats + V * H)

    def prefill_flops(T):
        return 2 * T * mats + att_flops_per_key * T * (T + 1) // 2 + rec_flops_per_token * T + 2 * V * H
    return weight_bytes, kv_per_token, state_bytes, prefill_flops


SOBEZEN_SIZES = {
    # name: (hidden, layers, heads, kv heads, head size, feed-forward, vocabulary)
    "2k": (2048, 8, 32, 8, 64, 8192, 32000),
    "4k": (4096, 4, 32, 8, 128, 14336, 32000),
}


def run_compare_sobezen(args):
    """Prefill and decode of Sobezen beside Llama, both with random weights, at equal hidden size, number of layers,
    heads, head size, feed-forward width (three matrices in both) and vocabulary: one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    names = [n for n in SOBEZEN_SIZES if not args.sizes or n in args.sizes.split(",")]
    for name in names:
        hidden, runs, heads, kv, dim, ff, vocab = SOBEZEN_SIZES[name]
        llama = dict(LLAMA_1B, num_hidden_layers=runs, hidden_size=hidden, num_attention_heads=heads, num_key_value_heads=kv,
                     head_dim=dim, intermediate_size=ff, vocab_size=vocab, tie_word_embeddings=False, rope_scaling=None)
        zen = sobezen_config(hidden, runs, heads, kv, dim, ff, vocab)
        for label, cfg in (("llama", llama), ("sobezen", zen)):
            if args.model and args.model != label:
                continue
            state_bytes = 0
            if label == "llama":
                wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
            else:
                wbytes, kv_per_tok, state_bytes, flops_fn = sobezen_numbers(cfg)
            flops = flops_fn(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            step_bytes = wbytes + args.batch * (ctx_len * kv_per_tok + state_bytes)
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "layers": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "order": [L["type"] for L in zen["layers"]] if label == "sobezen" else None},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": round(step_bytes / 1e9, 3),
                                         "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


# ---------------------------------------------------------------- Tazizen beside Llama at equal sizes
def tazizen_config(hidden, runs, heads, kv, dim, ff, vocab, streams=4, window=1024, kv_rank=512, experts=32, top=4):
    """A Tazizen model of `runs` layers in the order latent attention, latent attention, attention, every layer with the
    routed feed-forward: `experts` experts of ff / 8 of which `top` (4: half of ff) are chosen among the better half of
    four groups, and a shared expert of ff / 2, so that a token uses as many feed-forward values as Llama's dense one.
    `streams` copies of the residual stream; windows of `window` positions everywhere.  The latent layers' heads have
    `dim` unrotated and dim / 2 rotated channels and a query latent of 3 / 8 of the width."""
    rot = dict(dims=dim, base=1e4, scaling=dict(factor=4.0, original=2048, fast=32.0, slow=1.0))
    rot_l = dict(dims=dim // 2, base=1e6)
    mlp = dict(kind="moe", expert=dict(ff=ff // 8), shared=dict(ff=ff // 2),
               router=dict(experts=experts, top=top, scale=1.5, groups=dict(count=4, keep=2)))
    layers = []
    for i in range(runs):
        if i % 3 == 2:
            L = dict(type="attention", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, rot=rot, mask=dict(size=window)))
        else:
            L = dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=dim // 2, vdim=dim, kv_rank=kv_rank, q_rank=hidden * 3 // 8,
                                                         scale=(dim + dim // 2) ** -0.5, rot=rot_l, mask=dict(size=window)))
        layers.append(dict(mlp=mlp, **L))
    return dict(architecture="Tazizen", vocab=vocab, width=hidden, norm=dict(eps=1e-5), streams=streams, layers=layers)


def tazizen_numbers(c, batch):
    """(bytes a decode step of `batch` sequences reads apart from the cache, cache bytes per visible token and layer kind
    as a function of the context, prefill flops of T tokens with one wanted row)."""
    H, V = c["width"], c["vocab"]
    used, touched, per_key = 0, 0, []                 # matrix values a token uses / a decode step can touch
    for L in c["layers"]:
        m = L["mixer"]
        window = (m.get("mask") or {}).get("size") or (1 << 30)
        if L["type"] == "attention":
            mats = H * (m["heads"] * (m["dim"] + m["vdim"]) + m["kv_heads"] * (m["dim"] + m["vdim"])) + m["heads"] * m["vdim"] * H
            per_key.append((window, 2 * m["kv_heads"] * (m["dim"] + m["vdim"]), 2 * m["heads"] * (m["dim"] + m["vdim"])))
        else:
            row = m["kv_rank"] + m["rot_dim"]
            mats = H * m["q_rank"] + m["q_rank"] * m["heads"] * (m["dim"] + m["rot_dim"]) + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"]
            mats += m["heads"] * m["vdim"] * H + H * row
            per_key.append((window, 2 * row, 2 * m["heads"] * (row + m["kv_rank"])))
        used += mats
        touched += mats
        f = L["mlp"]
        if f:
            r, one = f["router"], 3 * H * f["expert"]["ff"]
            shared = 3 * H * f["shared"]["ff"] + H if f.get("shared") else 0
            used += r["experts"] * H + r["top"] * one + shared
            touched += r["experts"] * H + min(r["experts"], batch * r["top"]) * one + shared
    weight_bytes = 2 * (touched + V * H)

    def cache_bytes(ctx_len):
        return sum(b * min(ctx_len, w) for w, b, _ in per_key)

    def prefill_flops(T):
        att = sum(fl * sum(min(p + 1, w) for p in range(T)) for w, _, fl in per_key)
        return 2 * T * used + att + 2 * V * H
    return weight_bytes, cache_bytes, prefill_flops


def run_compare_tazizen(args):
    """Prefill and decode of Tazizen beside Llama, both with random weights, at equal hidden size, number of layers,
    heads, head size, feed-forward values used per token and vocabulary: one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    names = [n for n in SOBEZEN_SIZES if not args.sizes or n in args.sizes.split(",")]
    for name in names:
        hidden, runs, heads, kv, dim, ff, vocab = SOBEZEN_SIZES[name]
        llama = dict(LLAMA_1B, num_hidden_layers=runs, hidden_size=hidden, num_attention_heads=heads, num_key_value_heads=kv,
                     head_dim=dim, intermediate_size=ff, vocab_size=vocab, tie_word_embeddings=False, rope_scaling=None)
        zen = tazizen_config(hidden, runs, heads, kv, dim, ff, vocab)
        for label, cfg in (("llama", llama), ("tazizen", zen)):
            if args.model and args.model != label:
                continue
            if label == "llama":
                wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
                cache_fn = lambda n: n * kv_per_tok
            else:
                wbytes, cache_fn, flops_fn = tazizen_numbers(cfg, args.batch)
            flops = flops_fn(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            step_bytes = wbytes + args.batch * cache_fn(ctx_len)
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "layers": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "order": [L["type"] for L in zen["layers"]] if label == "tazizen" else None,
                                         "streams": zen["streams"] if label == "tazizen" else None},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": round(step_bytes / 1e9, 3),
                                         "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


# ---------------------------------------------------------------- Fomodra beside Tazizen at equal sizes
def fomodra_config(hidden, runs, heads, kv, dim, ff, vocab, window=1024, kv_rank=512, experts=32, identity=4, top=4):
    """A Fomodra model of `runs` layers in the order attention, parallel, latent attention, attention that borrows the first's keys
    and values, every layer with the routed feed-forward: `experts` experts of ff / 8 and `identity` identity experts, of which
    `top` (4: half of ff) are chosen, and a shared expert of ff / 2.  Windows and chunks of `window` positions; chunked attention with
    half the heads and values twice as wide as keys; a scan of 2 * hidden channels with 16 states, a dt input of hidden / 16; latent
    heads of dim unrotated and dim / 2 rotated channels; side vectors of hidden / 8."""
    rot, mask = dict(dims=dim, base=2.5e5), dict(size=window)
    mlp = dict(kind="moe", expert=dict(ff=ff // 8, limit=7.0), shared=dict(ff=ff // 2, limit=7.0),
               router=dict(experts=experts, identity=identity, top=top))
    att = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, rot=rot, mask=mask)
    left = dict(heads=heads // 2, kv_heads=kv // 2, dim=dim, vdim=2 * dim, scale=dim ** -0.5, mask=mask,
                rot=dict(dims=dim, base=5e5, scaling=dict(factor=4.0, low=1.0, high=4.0, original=2048)))
    layers = []
    for i in range(runs):
        if i % 4 == 1:
            L = dict(type="parallel", mixer=dict(left=left, right=dict(inner=2 * hidden, state=16, dt_rank=hidden // 16, conv=4)))
        elif i % 4 == 2:
            L = dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=dim // 2, vdim=dim, kv_rank=kv_rank, mask=mask,
                                                         scale=(dim + dim // 2) ** -0.5, rot=dict(dims=dim // 2, base=1e6)))
        else:
            L = dict(type="attention", mixer=dict(att, **({"kv_from": i - 3} if i % 4 == 3 else {})))
        layers.append(dict(mlp=mlp, **L))
    return dict(architecture="Fomodra", vocab=vocab, width=hidden, norm=dict(eps=1e-5), layers=layers, token_side=dict(dim=hidden // 8),
                embedding=dict(bigram=dict(buckets=50021, mul_prev=31337, mul_cur=7)))


def fomodra_numbers(c, batch):
    """(bytes a decode step reads at least and at most apart from cache and state: the experts that every sequence chooses alike, or
    that no two share; cache bytes of a sequence as a function of its length, bytes of state a step reads and writes per sequence,
    prefill flops of T tokens with one wanted row)."""
    H, V = c["width"], c["vocab"]
    used = most = state = rec = 0
    att = []                                          # (window or chunk, chunked, cache bytes a key, flops a key)
    for L in c["layers"]:
        m = L["mixer"]
        a = m["left"] if L["type"] == "parallel" else m
        size = (a.get("mask") or {}).get("size") or (1 << 30)
        if L["type"] == "latent_attention":
            row = m["kv_rank"] + m["rot_dim"]
            mats = H * m["heads"] * (m["dim"] + m["rot_dim"]) + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"] + m["heads"] * m["vdim"] * H
            mats += H * (row + m["heads"])
            att.append((size, False, 2 * row, 2 * m["heads"] * (m["dim"] + m["rot_dim"] + m["vdim"])))
        else:
            own = "kv_from" not in a
            mats = H * (a["heads"] * a["dim"] + (a["kv_heads"] * (a["dim"] + a["vdim"]) if own else 0)) + a["heads"] * a["vdim"] * H
            att.append((size, L["type"] == "parallel", 2 * a["kv_heads"] * (a["dim"] + a["vdim"]), 2 * a["heads"] * (a["dim"] + a["vdim"])))
        if L["type"] == "parallel":
            r = m["right"]
            I, N, R = r["inner"], r["state"], r["dt_rank"]
            mats += 3 * H * I + I * (R + 2 * N) + I * R
            state += 2 * 4 * I * (N + r["conv"] - 1)
            rec += 6 * I * N
            most += 4 * I * N                         # A_log, 32-bit
        mats += 2 * H * c["token_side"]["dim"]
        f = L["mlp"]
        r, one = f["router"], 3 * H * f["expert"]["ff"]
        fixed = mats + (r["experts"] + r["identity"]) * H + 3 * H * f["shared"]["ff"]
        used += fixed + r["top"] * one
        most += fixed + min(r["experts"], batch * r["top"]) * one

    def seen(p, size, chunked):
        return p % size + 1 if chunked else min(p + 1, size)

    def cache_bytes(n):
        return sum(b * seen(n - 1, w, ch) for w, ch, b, _ in att)

    def prefill_flops(T):
        return 2 * T * used + T * rec + sum(fl * sum(seen(p, w, ch) for p in range(T)) for w, ch, _, fl in att) + 2 * V * H
    return (2 * (used + V * H), 2 * (most + V * H)), cache_bytes, state, prefill_flops


def run_compare_fomodra(args):
    """Prefill and decode of Fomodra beside Tazizen (the other design with windowed and latent attention, corrected routing and a
    shared expert), both with random weights, at equal hidden size, number of layers, heads, head size, feed-forward values used per
    token and vocabulary: one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    for name in [n for n in SOBEZEN_SIZES if not args.sizes or n in args.sizes.split(",")]:
        hidden, runs, heads, kv, dim, ff, vocab = SOBEZEN_SIZES[name]
        for label in ("tazizen", "fomodra"):
            if args.model and args.model != label:
                continue
            if label == "tazizen":
                cfg, state = tazizen_config(hidden, runs, heads, kv, dim, ff, vocab), 0
                most, cache_fn, flops_fn = tazizen_numbers(cfg, args.batch)
                one = 2 * 3 * hidden * (ff // 8)
                r = cfg["layers"][0]["mlp"]["router"]
                wbytes = (most - runs * (min(r["experts"], args.batch * r["top"]) - r["top"]) * one, most)
            else:
                cfg = fomodra_config(hidden, runs, heads, kv, dim, ff, vocab)
                wbytes, cache_fn, state, flops_fn = fomodra_numbers(cfg, args.batch)
            flops = flops_fn(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            sampler = ClockSampler()
            sampler.start()
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            clocks = sampler.stop()
            step_bytes = [b + args.batch * (cache_fn(ctx_len) + state) for b in wbytes]
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "layers": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "order": [L["type"] for L in cfg["layers"]]},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": [round(b / 1e9, 3) for b in step_bytes],      # at least, at most
                                         "hbm_frac_at_least": round(step_bytes[0] / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "clocks": clocks, "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


def rarelorn_config(hidden, runs, heads, kv, dim, ff, vocab, window=1024, experts=32, top=4, taps=4):
    """A Rarelorn model of `runs` layer runs: [parallel, mlstm, delta, delta] as often as the runs ask for (a loop over the
    four layers), every layer with `experts` experts of ff / 4 of which `top` are chosen in the better half of four groups (a
    token uses as many feed-forward values as a dense one of ff).  Recurrent heads: hidden / dim of `dim` channels each."""
    mlp = dict(kind="moe", expert=dict(ff=ff // 4), router=dict(experts=experts, top=top, scale=2.0, groups=dict(count=4, keep=2)))
    left = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, conv=taps, scale=dim ** -0.5, softcap=20.0, rot=dict(dims=dim // 2, base=5e4),
                mask=dict(size=window))
    n = hidden // dim
    layers = [dict(type="parallel", mixer=dict(left=left, left_scale=0.9, right=dict(heads=n, dim=dim), right_scale=1.1)),
              dict(type="mlstm", mixer=dict(heads=n, dim=dim, vdim=dim, gate_cap=15.0))]
    layers += [dict(type="delta", mixer=dict(heads=n, kv_heads=n, dim=dim, vdim=dim, conv=taps))] * 2
    return dict(architecture="Rarelorn", vocab=vocab, width=hidden, norm=dict(eps=1e-5), layers=[dict(L, mlp=mlp) for L in layers],
                loop=dict(start=0, stop=4, times=max(1, runs // 4)))


def rarelorn_numbers(c, batch, rank=16):
    """(bytes a decode step of `batch` sequences reads at least and at most apart from cache and state: the experts that every
    sequence chooses alike, or that no two share; cache bytes of a sequence as a function of its length, bytes of state a step
    reads and writes per sequence, prefill flops of T tokens with one wanted row)."""
    H, V = c["width"], c["vocab"]
    loop = c["loop"]
    runs = list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], len(c["layers"])))
    used = most = state = rec = 0
    att = []                                          # (window, cache bytes a key, flops a key)
    for i in runs:
        m, kind = c["layers"][i]["mixer"], c["layers"][i]["type"]
        if kind == "parallel":
            l, r = m["left"], m["right"]
            W = r["heads"] * r["dim"]
            C = l["heads"] * l["dim"] + l["kv_heads"] * (l["dim"] + l["vdim"])
            mats = H * C + l["heads"] * l["vdim"] * H + 5 * H * W + rank * (H + 2 * W)
            att.append((l["mask"]["size"], 2 * l["kv_heads"] * (l["dim"] + l["vdim"]), 2 * l["heads"] * (l["dim"] + l["vdim"])))
            state += 2 * 4 * (r["heads"] * r["dim"] ** 2 + (l["conv"] - 1) * C)
            rec += 6 * r["heads"] * r["dim"] ** 2
        else:
            G = m.get("kv_heads", m["heads"])
            W = m["heads"] * m["vdim"]
            mats = H * (2 * G * m["dim"] + 3 * W + 2 * m["heads"])
            state += 2 * 4 * m["heads"] * m["dim"] * m["vdim"]
            if kind == "delta":
                state += 2 * 4 * (m["conv"] - 1) * (2 * G * m["dim"] + W)
            rec += (8 if kind == "delta" else 6) * m["heads"] * m["dim"] * m["vdim"]
        f = c["layers"][i]["mlp"]
        r, one = f["router"], 3 * H * f["expert"]["ff"]
        used += mats + r["experts"] * H + r["top"] * one
        most += mats + r["experts"] * H + min(r["experts"], batch * r["top"]) * one

    def cache_bytes(n):
        return sum(b * min(n, w) for w, b, _ in att)

    def prefill_flops(T):
        return 2 * T * used + T * rec + sum(fl * sum(min(p + 1, w) for p in range(T)) for w, _, fl in att) + 2 * V * H
    return (2 * (used + V * H), 2 * (most + V * H)), cache_bytes, state, prefill_flops


def run_compare_rarelorn(args):
    """Prefill and decode of Rarelorn beside Sesuzen (the other design with a recurrent state, windowed attention and routed
    experts), both with random weights, at equal hidden size, number of layer runs, heads, head size, feed-forward values
    used per token and vocabulary: one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    for name in [n for n in ("2k", "4k") if not args.sizes or n in args.sizes.split(",")]:
        hidden, runs, heads, kv, dim, ff, vocab, window, keep, _ = SESUZEN_SIZES[name]
        for label in ("sesuzen", "rarelorn"):
            if args.model and args.model != label:
                continue
            if label == "sesuzen":
                cfg = sesuzen_config(hidden, runs, heads, kv, dim, ff, vocab, window, keep)
                dense, kv_tok, state, flops_fn = sesuzen_numbers(cfg, args.batch)
                wbytes, cache_fn = (dense, dense), lambda n: kv_tok * min(n, window + keep)
            else:
                cfg = rarelorn_config(hidden, runs, heads, kv, dim, ff, vocab, window)
                wbytes, cache_fn, state, flops_fn = rarelorn_numbers(cfg, args.batch)
            flops = flops_fn(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            sampler = ClockSampler()
            sampler.start()
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            clocks = sampler.stop()
            step_bytes = [b + args.batch * (cache_fn(ctx_len) + state) for b in wbytes]
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "runs": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "window": window},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": [round(b / 1e9, 3) for b in step_bytes],      # at least, at most
                                         "hbm_frac_at_least": round(step_bytes[0] / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "clocks": clocks, "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


def run_compare(args):
    """Prefill and decode of Sinezen beside Llama, both with random weights, at equal hidden size, layer
    runs, heads, head size, feed-forward width (with experts: equal matrix values used per token) and
    vocabulary: one JSON line per size and model."""
    import torch
    from libllm_b200 import Model
    pk = peaks()
    names = [n for n in COMPARE_SIZES if not args.sizes or n in args.sizes.split(",")]
    for name in names:
        hidden, runs, heads, kv, dim, ff, vocab, mask, routed = COMPARE_SIZES[name]
        llama = dict(LLAMA_1B, num_hidden_layers=runs, hidden_size=hidden, num_attention_heads=heads, num_key_value_heads=kv,
                     head_dim=dim, intermediate_size=ff, vocab_size=vocab, tie_word_embeddings=False, rope_scaling=None)
        zen = sinezen_config(hidden, runs, heads, kv, dim, ff, vocab, mask, routed)
        for label, cfg in (("llama", llama), ("sinezen", zen)):
            if label == "llama":
                wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
                flops = flops_fn(PROMPT)
            else:
                wbytes, kv_per_tok, zen_flops = sinezen_numbers(cfg, args.batch)
                flops = zen_flops(PROMPT)
            model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=args.batch * CONTEXT, max_seq_len=CONTEXT)
            pre = prefill_rate(model, vocab, lambda T: flops, pk["bf16_tflops"])
            rate, ms, ctx_len, launches = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
            seen = ctx_len if label == "llama" else min(ctx_len, ctx_len % mask + 1)
            step_bytes = wbytes + args.batch * seen * kv_per_tok
            print(json.dumps({"compare": name, "model": label, "batch": args.batch, "prompt": PROMPT,
                              "config": {"hidden": hidden, "layer_runs": runs, "heads": heads, "kv_heads": kv, "head_dim": dim, "ff": ff,
                                         "vocab": vocab, "mask": mask if label == "sinezen" else None, "routed": routed if label == "sinezen" else None},
                              "prefill": {"ms": round(pre["ms"], 3), "tok_s": round(pre["value"], 1), "tflop": round(flops / 1e12, 3),
                                          "frac_of_gemm_peak": round(pre["frac"], 4)},
                              "decode": {"tok_s": round(rate, 1), "ms_per_step": round(ms, 4), "launches_per_step": launches,
                                         "step_gb": round(step_bytes / 1e9, 3),
                                         "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)},
                              "peaks": pk["source"]}), flush=True)
            model.engine.close()
            del model
            torch.cuda.empty_cache()
    return 0


def run_reference(args):
    """The reference arm: ling0322/libllm's unmodified C++/CUDA code (compiled into baseline/_ref by
    baseline/reference_arm.py; it has no installable Python package of its engine) at the same layer
    sizes, batch and prompt length, in its own compute type (float16), timed with a device
    synchronisation on both sides.  Where it cannot be built or run, one line says why."""
    def unavailable(why):
        print(json.dumps({"impl": "reference", "unavailable": " ".join(str(why).split())[:600]}))
        return 0
    if args.gpus != 1:
        return unavailable("ling0322/libllm runs on one GPU (every CUDA call of it targets device 0)")
    sys.path.insert(0, os.path.join(ROOT, "baseline"))
    try:
        import reference_arm
        reference_arm.build()
    except Exception as e:                       # no checkout, no compiler, a compile error
        return unavailable(f"the reference could not be compiled here: {e}")
    try:
        import torch
        if not torch.cuda.is_available():
            return unavailable("no CUDA device")
    except ImportError:
        pass
    cfg = dict(LLAMA_1B)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    warmup = max(args.warmup, 3)
    sampler = ClockSampler()
    sampler.start()
    try:
        r = reference_arm.run(cfg, PROMPT, args.batch, args.steps, warmup, CONTEXT)
    except Exception as e:
        sampler.stop()
        return unavailable(f"the reference's driver failed: {e}")
    clocks = sampler.stop()
    pk = peaks()
    wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
    ms, e2e_ms = r["decode_ms_per_step"], r["e2e_ms_per_step"]
    step_bytes = wbytes + args.batch * (PROMPT + warmup + args.steps // 2) * kv_per_tok
    achieved = step_bytes / (ms * 1e-3) / 1e9
    print(json.dumps({
        "metric": "decode tok/s (Llama-3.2-1B layer sizes, batch 8, 2048-token prompts, 4096 context)",
        "value": round(args.batch * 1000.0 / ms, 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "fp16", "data": "synthetic", "impl": "reference",
        "config": {"model": "llama-3.2-1b-sizes", "layers": cfg["num_hidden_layers"], "layers_full": full_layers,
                   "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                   "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
                   "global_batch": args.batch, "seq_len": CONTEXT, "prompt_len": PROMPT, "parallelism": "single-gpu",
                   "weights": "random fp16 N(0,0.02), tied", "attention": "the reference's portable path (FlashAttention off)",
                   "l2": "step reads more than L2 (no flush)", "peaks": pk["source"]},
        "e2e": {"value": round(args.batch * 1000.0 / e2e_ms, 1), "unit": "tok/s", "h2d_bytes_per_step": 8 * args.batch,
                "d2h_bytes_per_step": 8 * args.batch},
        "clocks": clocks,
        "prefill": {"value": round(PROMPT * 1000.0 / r["prefill_ms"], 1), "tokens": PROMPT, "ms": round(r["prefill_ms"], 4),
                    "frac": round(flops_fn(PROMPT) / (r["prefill_ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)}}))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the configuration (named in config)")
    ap.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    ap.add_argument("--workload", choices=["1b", "3b", "8b"], default="1b",
                    help="1b: the benchmark line (default); 3b, 8b: the larger workloads, a line of their own")
    ap.add_argument("--only", choices=["decode", "prefill"], default=None,
                    help="run one part only and print a short line (for profiling; not a bench record)")
    ap.add_argument("--compare", choices=["sinezen", "sesuzen", "sobezen", "tazizen", "rarelorn", "fomodra"], default=None,
                    help="Sinezen, Sesuzen, Sobezen or Tazizen beside Llama (Rarelorn beside Sesuzen, Fomodra beside Tazizen) at equal sizes: prefill and decode, a line per size and model (not a bench record)")
    ap.add_argument("--model", choices=["llama", "sesuzen", "sobezen", "tazizen", "rarelorn", "fomodra"], default=None,
                    help="with --compare sesuzen, sobezen, tazizen, rarelorn or fomodra: one of the two models only")
    ap.add_argument("--sizes", default=None, help="with --compare: which of the sizes (2k, 4k, 2k-routed), with commas")
    ap.add_argument("--prompt-len", type=int, default=None,
                    help="with --only: prompts of this many tokens instead of 2048 (the context grows to fit)")
    args = ap.parse_args()
    if args.prompt_len:
        if not args.only and not args.compare:
            print("bench.py: --prompt-len goes with --only (the record is taken at the sizes BASELINE.json names)")
            return 2
        global PROMPT, CONTEXT
        PROMPT = args.prompt_len
        CONTEXT = max(CONTEXT, PROMPT + 2048)
    if args.impl == "reference":
        return run_reference(args)
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    args.warmup = max(args.warmup, 3)
    if args.compare == "sesuzen":
        return run_compare_sesuzen(args)
    if args.compare == "sobezen":
        return run_compare_sobezen(args)
    if args.compare == "tazizen":
        return run_compare_tazizen(args)
    if args.compare == "rarelorn":
        return run_compare_rarelorn(args)
    if args.compare == "fomodra":
        return run_compare_fomodra(args)
    if args.compare:
        return run_compare(args)
    if args.workload != "1b":
        return run_workload(args)

    import torch
    from libllm_b200 import Model
    cfg = dict(LLAMA_1B)
    full_layers = cfg["num_hidden_layers"]
    if args.layers:
        cfg["num_hidden_layers"] = args.layers
    pk = peaks()
    wbytes, kv_per_tok, flops_fn = model_numbers(cfg)
    vocab = cfg["vocab_size"]
    max_batch = max(args.batch, 1 if (args.no_points or args.only) else 64)
    model = Model.from_random(cfg, seed=0, dtype="bfloat16", max_tokens=max_batch * CONTEXT, max_seq_len=CONTEXT)

    if args.only == "decode":
        rate, ms, ctx_len, _ = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
        step_bytes = wbytes + args.batch * ctx_len * kv_per_tok
        print(json.dumps({"only": "decode", "batch": args.batch, "tok_s": round(rate, 1), "ms_per_step": round(ms, 4),
                          "context": ctx_len, "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}))
        return 0
    if args.only == "prefill":
        print(json.dumps({"only": "prefill", **prefill_rate(model, vocab, flops_fn, pk["bf16_tflops"])}))
        return 0
    sampler = ClockSampler()
    sampler.start()
    rate, ms, ctx_len, launches_per_step = decode_rate(model, args.batch, args.steps, args.warmup, vocab)
    clocks = sampler.stop()
    step_times = sorted(LAST_STEP_TIMES)
    median_ms = step_times[len(step_times) // 2] if step_times else ms
    e2e, h2d, d2h = e2e_rate(model, args.batch, args.steps, args.warmup, vocab)
    prefill = prefill_rate(model, vocab, flops_fn, pk["bf16_tflops"])
    step_bytes = wbytes + args.batch * ctx_len * kv_per_tok
    achieved = step_bytes / (ms * 1e-3) / 1e9
    points = {}
    if not args.no_points:
        for b in (1, 64):
            r, _, _, _ = decode_rate(model, b, max(8, args.steps // 2), args.warmup, vocab)
            points[f"decode_b{b}"] = round(r, 1)
    line = {
        "metric": "decode tok/s (Llama-3.2-1B layer sizes, batch 8, 2048-token prompts, 4096 context)",
        "value": round(rate, 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "ms_per_step_median": round(median_ms, 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "ours",
        "config": {"model": "llama-3.2-1b-sizes", "layers": cfg["num_hidden_layers"], "layers_full": full_layers,
                   "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"],
                   "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
                   "intermediate": cfg["intermediate_size"], "vocab": vocab, "global_batch": args.batch,
                   "seq_len": CONTEXT, "prompt_len": PROMPT, "context_at_timing": ctx_len,
                   "parallelism": "single-gpu", "weights": "random bf16 N(0,0.02), tied",
                   "l2": "step reads more than L2 (no flush)", "peaks": pk["source"]},
        "e2e": {"value": round(e2e, 1), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h},
        "gpu_launches": launches_per_step * args.steps,
        "clocks": clocks,
        "prefill": {k: (round(v, 4) if isinstance(v, float) else v) for k, v in prefill.items()},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
        "dominant_kernel": products_alone(cfg, args.batch, pk),
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
