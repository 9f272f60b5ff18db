"""Comparisons shared by the tests of the served decoder families: the framework's sessions, scheduler and generation against
a family's plain statement of its equations."""
import json
import os

import torch

from litetorch_b200.models import registry
from litetorch_b200.serving import Request, ServingScheduler

TOL = {torch.float32: 1e-5, torch.bfloat16: 0.03}


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def server(eng, blocks=64, slots=4, block_size=16):
    return registry.new_serving(eng, num_blocks=blocks, block_size=block_size, max_num_seqs=slots), ServingScheduler(blocks, block_size, slots, 4096, -1)


def row_errors(got, want):
    """How far each row of logits is from what it should be (means taken off), relative to the size of all of them."""
    dlt = got.double().cpu() - want
    dlt = dlt - dlt.mean(-1, keepdim=True)
    return (dlt.pow(2).mean(-1) / want.var()).sqrt()


def error(got, want):
    """The larger of the root mean square over the rows and a third of the worst row."""
    row = row_errors(got, want)
    return max(float(row.pow(2).mean().sqrt()), float(row.max()) / 3.0)


def run_portions(model, sched, sid, toks, cuts):
    """Feed a sequence in portions of the given sizes (the last one repeats); logits at every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(sched.feed(model, [(sid, toks[at:at + n], list(range(n)))])[0])
        at += n
        k += 1
    return torch.cat(out)


def write_model(directory, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(directory, "model.safetensors"))
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)


class Suite:
    """configs: name -> configuration; weights(cfg, seed) -> tensors; engine(cfg, tensors, device, dtype); forward(cfg, tensors,
    tokens) -> logits of the plain statement; error(got, want, cfg, dtype) -> how far off, measured against TOL[dtype]."""

    def __init__(self, configs, weights, engine, forward, measure=None):
        self.configs, self.weights, self.engine, self.forward = configs, weights, engine, forward
        self.measure = measure or (lambda got, want, cfg, dtype: error(got, want))

    def reference(self, cfg, w, toks):
        with torch.no_grad():
            return self.forward(cfg, w, toks)

    def check_portions(self, name, device, dtype, length, schedules, block_size=16):
        """Whole prompts, portions and single tokens all give the logits of the plain statement."""
        cfg = self.configs[name]
        w = self.weights(cfg)
        toks = tokens(cfg, length, 1)
        want = self.reference(cfg, w, toks)
        model, sched = server(self.engine(cfg, w, device, dtype), blocks=2 * (length // block_size + 2), block_size=block_size)
        for n, cuts in enumerate(schedules):
            e = self.measure(run_portions(model, sched, n, toks, cuts), want, cfg, dtype)
            assert e < TOL[dtype], (name, cuts, e)
            sched.end_session(n)

    def check_interleaved(self, name, device, dtype):
        """Requests of unequal lengths in one step, prompts beside decoding, each against itself alone; then the pages and
        slots they leave are used by others."""
        cfg = self.configs[name]
        w = self.weights(cfg, 3)
        model, sched = server(self.engine(cfg, w, device, dtype), blocks=40, slots=4)
        free = sched.free_blocks
        for rnd in range(2):                                     # the second round meets the first one's cache and state
            lens = [70, 9, 41, 100] if rnd == 0 else [12, 97, 60, 33]
            seqs = [tokens(cfg, n, 10 * rnd + i) for i, n in enumerate(lens)]
            want = [self.reference(cfg, w, s) for s in seqs]
            at, got = [0] * 4, [[] for _ in range(4)]
            step = 0
            while any(at[i] < lens[i] for i in range(4)):
                entries = []
                for i in range(4):
                    n = min([1, 1, 5, 1, 2, 1, 17][(step + 2 * i) % 7] if step else lens[i] // 3, lens[i] - at[i])
                    if n:
                        entries.append((100 + i, seqs[i][at[i]:at[i] + n], list(range(n))))
                        at[i] += n
                for (sid, _, _), y in zip(entries, sched.feed(model, entries)):
                    got[sid - 100].append(y.cpu())
                step += 1
            for i in range(4):
                e = self.measure(torch.cat(got[i]), want[i], cfg, dtype)
                assert e < TOL[dtype], (name, rnd, i, e)
                sched.end_session(100 + i)
            assert sched.free_blocks == free

    def check_generate(self, name, device, dtype, max_new, budget):
        """Greedy generation through the scheduler: every token is the argmax of the plain statement's logits, up to rounding."""
        from litetorch_b200.models.serving_base import generate
        cfg = self.configs[name]
        w = self.weights(cfg, 5)
        prompts = [tokens(cfg, n, 40 + n) for n in (1, 2, 30, 75)]
        outs = generate(self.engine(cfg, w, device, dtype), prompts, max_new, max_num_seqs=3, max_num_batched_tokens=budget)
        for p, o in zip(prompts, outs):
            assert len(o) == max_new
            y = self.reference(cfg, w, p + o[:-1])[len(p) - 1:]
            gap = y.max(-1).values - y[torch.arange(max_new), torch.tensor(o)]
            assert float(gap.max() / y.std()) < 5 * TOL[dtype], (name, len(p), float(gap.max()))

    def check_generate_matches_decode_of_requests(self, name, device, dtype):
        """Requests that join and leave a running batch of the scheduler see each other in nothing."""
        cfg = self.configs[name]
        w = self.weights(cfg, 6)
        eng = self.engine(cfg, w, device, dtype)

        def run(prompts, slots):
            model = registry.new_serving(eng, num_blocks=64, max_num_seqs=slots)
            sched = ServingScheduler(64, 16, slots, 24, -1)
            reqs = [Request(i, p, max_new_tokens=4 + 3 * i) for i, p in enumerate(prompts)]
            for r in reqs:
                sched.add_request(r)
            done = []
            while len(done) < len(reqs):
                done += sched.step(model)
            assert sched.free_blocks == 64
            return [r.generated_tokens for r in reqs]

        prompts = [tokens(cfg, n, n) for n in (50, 3, 21, 34, 8)]
        assert run(prompts, 2) == run(prompts, 5)
