"""Small Safuvik models and comparisons shared by the CPU and the GPU tests: the framework's sessions, scheduler and
generation against the plain statement in `safuvik_ref`."""
import json
import os

import torch

import safuvik_ref as R
from litetorch_b200.models import registry
from litetorch_b200.models.safuvik import SafuvikConfig, SafuvikEngine, random_tensor, tensor_shapes
from litetorch_b200.serving import Request, ServingScheduler


def attention(heads, kv, dim, vdim, window, dims, scale=None, base=700.0, yarn=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale or dim ** -0.5,
            "rot": dict({"base": base, "dims": dims}, **({"scaling": yarn} if yarn else {}))}


def parallel(left, width, blocks, conv, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}}, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(vocab, width, streams, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Safuvik", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": layers}


CONFIGS = {
    # unequal sizes everywhere, a layer without feed-forward, window below and above a page, YaRN with a short original context
    "mixed": config(131, 96, 3, [
        mlstm(3, 20, 28, 5.0, None),
        parallel(attention(4, 2, 24, 40, 37, 12, yarn={"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}), 80, 5, 3, dense(72, 0.7)),
        parallel(attention(2, 2, 40, 24, 16, 40, scale=0.3, base=50.0), 48, 1, 2, None)], eps=1e-4, logit_scale=0.7),
    # sizes the tensor-core kernels take: heads of 128, gate blocks of 64, a window just over a tile
    "tiles": config(256, 128, 2, [
        parallel(attention(8, 2, 128, 64, 129, 32, yarn={"factor": 8.0, "original": 256, "fast": 16.0, "slow": 2.0}), 128, 2, 4, dense(192, 2.0)),
        mlstm(2, 64, 128, 9.0, dense(128, 1.2)),
        parallel(attention(4, 4, 64, 64, 200, 64), 256, 2, 5, dense(64, 3.0))], logit_scale=1.5),
    # nothing is a multiple of 8, one stream, no taps but the current one, many query heads on one key head
    "odd": config(77, 60, 1, [
        parallel(attention(17, 1, 10, 6, 23, 4), 33, 3, 1, dense(35, 0.5)),
        mlstm(1, 7, 5, 3.0, dense(21, 1.0)),
        mlstm(2, 70, 66, 12.0, None)], eps=1e-3),
    # head sizes beyond the tensor-core kernels, five streams
    "wide": config(64, 64, 5, [
        parallel(attention(2, 1, 144, 160, 50, 100, base=2000.0), 64, 1, 6, dense(48, 1.0)),
        mlstm(2, 130, 132, 6.0, dense(48, 1.0))]),
}


def weights(cfg, seed=0):
    """bf16 tensors.  Some queries and keys are scaled so that single scores stand out, which a wrong key, a window that is
    off by one or a wrong rotation cannot hide behind."""
    gen = torch.Generator().manual_seed(seed)
    w = {n: random_tensor(n, s, gen) for n, s in tensor_shapes(SafuvikConfig.parse(cfg)).items()}
    for n in w:
        if n.endswith(("q.norm", "k.norm")):
            w[n] = (w[n].float() * 2.0).to(torch.bfloat16)
    return w


def engine(cfg, w, device, dtype):
    return SafuvikEngine(SafuvikConfig.parse(cfg), w, device, dtype)


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def server(eng, blocks=64, slots=4, block_size=16):
    return registry.new_serving(eng, num_blocks=blocks, block_size=block_size, max_num_seqs=slots), ServingScheduler(blocks, block_size, slots, 4096, -1)


def reference(cfg, w, toks):
    with torch.no_grad():
        return R.forward(cfg, w, toks)


def error(got, want):
    """How far rows of logits are from what they should be (means taken off), relative to the size of all of them: the larger
    of the root mean square over the rows and a third of the worst row."""
    dlt = got.double().cpu() - want
    dlt = dlt - dlt.mean(-1, keepdim=True)
    row = dlt.pow(2).mean(-1) / want.var()
    return max(float(row.mean().sqrt()), float(row.max().sqrt()) / 3.0)


def run_portions(model, sched, sid, toks, cuts):
    """Feed a sequence in portions of the given sizes (the last one repeats); logits at every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(sched.feed(model, [(sid, toks[at:at + n], list(range(n)))])[0])
        at += n
        k += 1
    return torch.cat(out)


TOL = {torch.float32: 1e-5, torch.bfloat16: 0.03}


def check_portions(name, device, dtype, length, schedules):
    """Whole prompts, portions and single tokens all give the logits of the plain statement."""
    cfg = CONFIGS[name]
    w = weights(cfg)
    toks = tokens(cfg, length, 1)
    want = reference(cfg, w, toks)
    model, sched = server(engine(cfg, w, device, dtype), blocks=2 * (length // 16 + 2))
    for n, cuts in enumerate(schedules):
        e = error(run_portions(model, sched, n, toks, cuts), want)
        assert e < TOL[dtype], (name, cuts, e)
        sched.end_session(n)


def check_interleaved(name, device, dtype):
    """Requests of unequal lengths in one step, prompts beside decoding, each against itself alone; then the pages and
    slots they leave are used by others."""
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    model, sched = server(engine(cfg, w, device, dtype), blocks=40, slots=4)
    free = sched.free_blocks
    for rnd in range(2):                                     # the second round meets the first one's cache and state
        lens = [70, 9, 41, 100] if rnd == 0 else [12, 97, 60, 33]
        seqs = [tokens(cfg, n, 10 * rnd + i) for i, n in enumerate(lens)]
        want = [reference(cfg, w, s) for s in seqs]
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
            e = error(torch.cat(got[i]), want[i])
            assert e < TOL[dtype], (name, rnd, i, e)
            sched.end_session(100 + i)
        assert sched.free_blocks == free


def check_generate(name, device, dtype, max_new, budget):
    """Greedy generation through the scheduler: every token is the argmax of the plain statement's logits, up to rounding."""
    from litetorch_b200.models.serving_base import generate
    cfg = CONFIGS[name]
    w = weights(cfg, 5)
    prompts = [tokens(cfg, n, 40 + n) for n in (1, 2, 30, 75)]
    outs = generate(engine(cfg, w, device, dtype), prompts, max_new, max_num_seqs=3, max_num_batched_tokens=budget)
    for p, o in zip(prompts, outs):
        assert len(o) == max_new
        y = reference(cfg, w, p + o[:-1])[len(p) - 1:]
        gap = y.max(-1).values - y[torch.arange(max_new), torch.tensor(o)]
        assert float(gap.max() / y.std()) < 5 * TOL[dtype], (name, len(p), float(gap.max()))


def check_generate_matches_decode_of_requests(device, dtype):
    """Requests that join and leave a running batch of the scheduler see each other in nothing."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 6)
    eng = engine(cfg, w, device, dtype)

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


def write_model(directory, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(directory, "model.safetensors"))
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
