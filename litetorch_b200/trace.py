"""Replay a trace of token ids through a served model and write the logits it asks for (`bin/trace_run`).

    trace_run --model DIR --dtype bfloat16 --out DIR --max-tokens 4096 < steps.jsonl

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings a request's next tokens; "want" lists the places among them whose logits are written, in the order of the
entries, to OUT/<step>.f32 (little-endian fp32, [wanted, vocab]; no file for a step that wants nothing).  "end" lists
requests whose cache and state are given back after the step.  After every step a line "done <step>" is printed.

This is `ServingScheduler.feed` on the model that `models.registry` picks for the directory: the loader, the cache, the
state slots, the prompt and the decode step are those of generation.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def replay(model, sched, lines, out_dir: str, say=print) -> None:
    import numpy as np
    import torch
    ids = {}                                             # request name -> session id; a name may come again after its end
    fresh = 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in ids:
                ids[e["id"]] = fresh
                fresh += 1
            entries.append((ids[e["id"]], e["tokens"], e.get("want") or []))
        logits = [t for t, e in zip(sched.feed(model, entries), entries) if e[2]]
        if logits:
            a = torch.cat(logits).float().cpu().numpy().astype("<f4")
            path = os.path.join(out_dir, "%d.f32" % step["step"])
            np.ascontiguousarray(a).tofile(path + ".part")
            os.replace(path + ".part", path)
        for name in step.get("end") or []:
            if name in ids:
                sched.end_session(ids.pop(name))
        say("done %d" % step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a served model.")
    ap.add_argument("--model", required=True, help="directory with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=8, help="most requests alive at any time")
    ap.add_argument("--block-size", type=int, default=16)
    ap.add_argument("--device", default="cuda")
    args = ap.parse_args(argv)

    import torch
    from . import _native
    from .models import registry
    dtype = getattr(torch, args.dtype)
    fam = registry.family_of(registry.read_config(args.model))
    if args.device != "cpu":
        if dtype not in fam.dtypes:
            print("%s does not run in %s" % (fam.name, args.dtype), file=sys.stderr)
            return 3
        _native.ensure_cuda(fam.components)
    from .serving import ServingScheduler
    engine = registry.load_engine(args.model, args.device, dtype)
    blocks = (args.max_tokens + args.block_size - 1) // args.block_size + args.max_seqs     # every request may leave part of a block
    model = registry.new_serving(engine, num_blocks=blocks, block_size=args.block_size, max_num_seqs=args.max_seqs)
    sched = ServingScheduler(blocks, args.block_size, args.max_seqs, args.max_tokens)
    os.makedirs(args.out, exist_ok=True)
    replay(model, sched, sys.stdin, args.out, say=lambda s: print(s, flush=True))
    if engine.device.type == "cuda":
        from .ops import kernels as K
        K.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
