"""Safuvik on the CPU twin of the kernels (fp32): configuration, loading, portions, sessions, scheduler, trace replay."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import safuvik_ref as R
import safuvik_suite as U

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_portions_of_all_sizes_match_the_plain_statement(name):
    U.check_portions(name, "cpu", F32, 90, [[90], [2], [1], [7, 2, 30, 1, 1, 3, 16], [64, 1]])


def test_requests_side_by_side_and_reused_pages_and_slots():
    U.check_interleaved("mixed", "cpu", F32)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(name):
    U.check_generate(name, "cpu", F32, 6, 16)


def test_requests_that_share_a_batch_do_not_see_each_other():
    U.check_generate_matches_decode_of_requests("cpu", F32)


def test_frequencies_with_and_without_scaling():
    from litetorch_b200.models.safuvik import RotaryConfig
    for rot in ({"base": 300.0, "dims": 20}, {"base": 10.0, "dims": 6, "scaling": {"factor": 3.0, "original": 128, "fast": 4.0, "slow": 0.5}},
                {"base": 5e5, "dims": 64, "scaling": {"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}}):
        freq, gain = RotaryConfig.parse(rot).frequencies()
        want, want_gain = R.inverse_frequencies(rot)
        assert gain == want_gain and torch.allclose(torch.tensor(freq, dtype=torch.float64), want, rtol=1e-14)
    assert RotaryConfig.parse({"base": 5e5, "dims": 64, "scaling": {"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}}).frequencies()[0][-1] < 1e-6


def test_window_attention_twin_at_the_edges():
    """Keys that dominate just inside and just outside the window."""
    from litetorch_b200.ops import kernels_ref as K
    g = torch.Generator().manual_seed(0)
    T, H, G, D, E, window = 150, 4, 2, 16, 24, 33
    q, k, v = (torch.randn(T, n, m, generator=g) for n, m in ((H, D), (G, D), (G, E)))
    for t, gap in ((140, window - 1), (120, window), (60, window - 1), (100, window), (33, 32), (34, 34)):
        k[t - gap] = 6.0 * q[t].view(G, H // G, D)[:, 0]                # key `gap` back stands out for query t
    want = R.window_attention(q.double(), k.double(), v.double(), 0.25, window)
    o, _ = K.flash_fwd(q[None], k[None], torch.nn.functional.pad(v, (0, 0))[None], causal=True, scale=0.25, window=window)
    assert torch.allclose(o[0].double(), want, atol=1e-5)
    from litetorch_b200.serving import PagedKVCache
    cache = PagedKVCache.per_layer([(G, D, E)], 16, 16, "cpu", F32)
    table = torch.randperm(16, generator=g)[:10].int()
    pos = torch.arange(T)
    cache.append(0, k, v, (table.long()[pos // 16] * 16 + pos % 16).int())
    o = K.window_attn(q, cache.k[0], cache.v[0], table, pos.int(), D=D, E=E, window=window, scale=0.25)
    assert torch.allclose(o.double(), want, atol=1e-5)


def test_a_checkpoint_that_does_not_fit_is_refused(tmp_path):
    from litetorch_b200.models import registry
    cfg = U.CONFIGS["odd"]
    w = U.weights(cfg)
    d = str(tmp_path / "m")
    U.write_model(d, cfg, w)
    assert registry.load_engine(d, "cpu").cfg.vocab == cfg["vocab"]
    with pytest.raises(ValueError, match="l1.mix.q"):
        U.engine(cfg, dict(w, **{"l1.mix.q": w["l1.mix.q"][:, :-1]}), "cpu", F32)
    with pytest.raises(KeyError, match="l0.mix.right.lam"):
        U.engine(cfg, {k: t for k, t in w.items() if k != "l0.mix.right.lam"}, "cpu", F32)
    with pytest.raises(ValueError, match="unknown type"):
        U.SafuvikConfig.parse(dict(cfg, layers=[{"type": "other", "mixer": {}, "mlp": None}]))
    with pytest.raises(ValueError, match="no model family"):
        registry.family_of({"architecture": "Unheard"})
    with pytest.raises(TypeError):
        registry.new_serving(object(), num_blocks=4)


def test_a_pool_that_is_too_small_refuses_the_session():
    cfg = U.CONFIGS["odd"]
    model, sched = U.server(U.engine(cfg, U.weights(cfg), "cpu", F32), blocks=4, slots=2)
    sched.feed(model, [(1, U.tokens(cfg, 40, 0), [])])
    with pytest.raises(RuntimeError, match="too small"):
        sched.feed(model, [(2, U.tokens(cfg, 40, 0), [])])
    with pytest.raises(RuntimeError, match="slot"):
        sched.feed(model, [(3, [1], [])])
    for s in (1, 2):
        sched.end_session(s)
    assert sched.free_blocks == 4


def test_trace_replay(tmp_path):
    from litetorch_b200 import trace
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, 8)
    U.write_model(str(tmp_path / "m"), cfg, w)
    a, b = U.tokens(cfg, 50, 1), U.tokens(cfg, 30, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[20:21], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [27, 3]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "b", "tokens": a[:9], "want": [8]}, {"id": "a", "tokens": a[21:], "want": [28]}], "end": ["a", "b"]}]
    said = []
    from litetorch_b200.models import registry
    from litetorch_b200.serving import ServingScheduler
    model = registry.new_serving(registry.load_engine(str(tmp_path / "m"), "cpu"), num_blocks=8, max_num_seqs=2)
    trace.replay(model, ServingScheduler(8, 16, 2, 64), io.StringIO("\n".join(map(json.dumps, steps))), str(tmp_path), said.append)
    assert said == ["done %d" % i for i in range(4)] and not os.path.exists(str(tmp_path / "1.f32"))
    ya, yb = U.reference(cfg, w, a), U.reference(cfg, w, b)
    want = {0: ya[[0, 19]], 2: torch.stack([ya[20], yb[29], yb[5]]), 3: ya[[8, 49]]}
    for n, y in want.items():
        got = torch.from_numpy(np.fromfile(str(tmp_path / ("%d.f32" % n)), dtype="<f4")).view(len(y), -1)
        assert U.error(got, y) < 1e-5


def test_trace_program_on_the_cpu(tmp_path):
    cfg = U.CONFIGS["odd"]
    U.write_model(str(tmp_path / "m"), cfg, U.weights(cfg))
    line = json.dumps({"step": 7, "entries": [{"id": "x", "tokens": [1, 2, 3], "want": [2]}], "end": ["x"]})
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--out", str(tmp_path), "--dtype", "float32", "--max-tokens", "64",
           "--device", "cpu"]
    r = subprocess.run(cmd, input=line + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and "done 7" in r.stdout.splitlines(), r.stderr[-2000:]
    assert os.path.getsize(str(tmp_path / "7.f32")) == 4 * cfg["vocab"]
    # a family without fp32 kernels says so before it loads anything
    from litetorch_b200 import trace
    os.makedirs(str(tmp_path / "llama"))
    with open(str(tmp_path / "llama" / "config.json"), "w") as f:
        json.dump({"model_type": "llama"}, f)
    assert trace.main(["--model", str(tmp_path / "llama"), "--out", str(tmp_path), "--dtype", "float32"]) == 3


def test_generation_example_on_a_directory(tmp_path):
    cfg = U.CONFIGS["odd"]
    w = U.weights(cfg, 2)
    U.write_model(str(tmp_path / "m"), cfg, w)
    sys.path.insert(0, os.path.join(ROOT, "examples"))
    import generate_llama
    res = generate_llama.main(["--model", str(tmp_path / "m"), "--prompt", "5,6,7", "--ids", "--max-new-tokens", "5", "--device", "cpu"])
    seq = [5, 6, 7]
    for t in res["outputs"][0]:
        assert t == int(U.reference(cfg, w, seq)[-1].argmax())
        seq.append(t)
    warm = generate_llama.main(["--model", str(tmp_path / "m"), "--prompt", "5,6,7", "--ids", "--max-new-tokens", "5", "--device", "cpu",
                                "--temperature", "0.9", "--top-k", "8", "--seed", "3"])
    assert len(warm["outputs"][0]) == 5
