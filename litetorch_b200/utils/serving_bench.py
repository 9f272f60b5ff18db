"""Timing of served models and of single kernels, shared by the comparisons of a decoder family with Llama models of equal
size: weights are random; prompts are one sequence through `prefill_chunk`, decoding is one step of B sequences (CUDA-graph
replay), both timed with CUDA events after warm-up; kernels are replayed from a graph one call at a time with the L2
overwritten before each call, against max(bytes / measured copy bandwidth, FLOPs / measured bf16 GEMM rate).
"""
from __future__ import annotations

import argparse
import json
import os

import torch


def llama_config(size: str, params: int):
    """The Llama shape of that size with as many layers as come closest to `params` parameters."""
    import dataclasses

    from ..models.llama import LlamaConfig
    base = LlamaConfig.llama_1b() if size == "1b" else LlamaConfig.llama3_8b()
    base = dataclasses.replace(base, vocab_size=32000, max_seq=1 << 15)
    one = dataclasses.replace(base, n_layers=1).num_params() - dataclasses.replace(base, n_layers=0).num_params()
    n = round((params - dataclasses.replace(base, n_layers=0).num_params()) / one)
    return dataclasses.replace(base, n_layers=n)


def peaks():
    """(copy bytes/s, bf16 FLOP/s) as measured on this machine, else an earlier measurement of the same hardware."""
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]) * 1e9, float(p["bf16_tflops"]) * 1e12
    except (OSError, KeyError, ValueError, TypeError):
        return 6.65e12, 1.59e15


def event_ms(fn, warm=3, steps=10, flush=None) -> float:
    """Median device time of a call."""
    times = []
    for i in range(warm + steps):
        if flush is not None:
            flush.add_(1)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warm:
            times.append(a.elapsed_time(b))
    return sorted(times)[len(times) // 2]


def graph_ms(fn, flush) -> float:
    """Device time of a call replayed from a CUDA graph (no launch gaps between its kernels), cold L2."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=side):
        fn()
    return event_ms(g.replay, flush=flush)


def throughput(serving_of, cfg_name, params, vocab, prompt, context, batches, out):
    bs = 16
    for kind, B in [("prefill", 1)] + [("decode", b) for b in batches]:
        n = prompt if kind == "prefill" else context + 16
        per = (n + bs - 1) // bs + 1
        model = serving_of(B * per, B)
        for t in model.cache.k + model.cache.v:
            if t is not None:
                t.normal_()
        slots = {} if not model.state_slots else {"slot": 0} if kind == "prefill" else {"slots": list(range(B))}
        tables = [list(range(s * per, (s + 1) * per)) for s in range(B)]
        if kind == "prefill":
            toks = [(7 * i) % vocab for i in range(prompt)]
            ms = event_ms(lambda: model.prefill_chunk(toks, 0, tables[0], True, **slots))
            rate = prompt / ms * 1e3
        else:
            ms = event_ms(lambda: model.decode_batch([1] * B, [context] * B, tables, **slots))
            rate = B / ms * 1e3
        row = {"model": cfg_name, "params": params, "work": kind, "batch": B, "tokens": prompt if kind == "prefill" else context, "ms": round(ms, 3),
               "tokens_per_s": round(rate, 1)}
        print(json.dumps(row), flush=True)
        out.append(row)
        del model
        torch.cuda.empty_cache()


def llama_throughput(size, params, prompt, context, batches, out):
    from ..models.llama_serving import LlamaKVModel
    from .decode_bench import inference_engine
    lc = llama_config(size, params)
    le = inference_engine(lc)
    throughput(lambda nb, B: LlamaKVModel(le, num_blocks=nb), "llama-" + size, lc.num_params(), lc.vocab_size, prompt, context, batches, out)


class KernelTable:
    """Rows (group, design, name, ms, floor ms); a group holds like kernels of the designs."""

    def __init__(self, size):
        self.size, self.rows = size, []
        self.hbm, self.mma = peaks()
        self.flush = torch.zeros(64 << 20, device="cuda")

    def add(self, group, design, name, fn, nbytes=0.0, flops=0.0):
        ms = graph_ms(fn, self.flush)
        floor = max(nbytes / self.hbm, flops / self.mma) * 1e3
        self.rows.append((group, design, name, ms, floor))
        print(json.dumps({"size": self.size, "group": group, "design": design, "kernel": name, "us": round(ms * 1e3, 1), "floor_us": round(floor * 1e3, 1),
                          "fraction": round(floor / ms, 3)}), flush=True)


def tables(models, kernels):
    out = ["| model | parameters | work | batch | tokens | ms | tokens/s |", "|---|---|---|---|---|---|---|"]
    for m in models:
        out.append("| %s | %.2f B | %s | %d | %d | %.3f | %.0f |" % (m["model"], m["params"] / 1e9, m["work"], m["batch"], m["tokens"], m["ms"], m["tokens_per_s"]))
    for size, rows in kernels:
        out += ["", "%s layers:" % size, "", "| kernel | design | us | floor us | fraction |", "|---|---|---|---|---|"]
        for g, design, name, ms, floor in rows:
            out.append("| %s: %s | %s | %.1f | %.1f | %.2f |" % (g, name, design, ms * 1e3, floor * 1e3, floor / ms))
    return "\n".join(out)


def run(argv, compare_models, compare_kernels):
    """The command line of a comparison: compare_models(size, prompt, context, batches) and compare_kernels(size, prompt, context,
    batch), each returning rows."""
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="1b,8b-layers")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--batches", default="1,32")
    ap.add_argument("--parts", default="models,kernels")
    a = ap.parse_args(argv)
    from ..ops import kernels as K
    torch.cuda.set_device(0)
    models, kernels = [], []
    for size in a.sizes.split(","):
        if "kernels" in a.parts:
            kernels.append((size, compare_kernels(size, a.prompt, a.context, max(int(b) for b in a.batches.split(",")))))
        if "models" in a.parts:
            models += compare_models(size, a.prompt, a.context, [int(b) for b in a.batches.split(",")])
    K.check_status()
    print(tables(models, kernels))
