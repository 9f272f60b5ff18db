"""Ravenex on the CPU twin of the kernels (fp32): configuration, loading, portions, sessions, scheduler, trace replay."""
import copy
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ravenex_ref as R
import ravenex_suite as U

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_portions_of_all_sizes_match_the_plain_statement(name):
    U.SUITE.check_portions(name, "cpu", F32, 90, [[90], [2], [1], [7, 2, 30, 1, 1, 3, 16], [64, 1]])


@pytest.mark.parametrize("name", ["mixed", "choice"])
def test_requests_side_by_side_and_reused_pages(name):
    U.SUITE.check_interleaved(name, "cpu", F32)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(name):
    U.SUITE.check_generate(name, "cpu", F32, 6, 16)


def test_requests_that_share_a_batch_do_not_see_each_other():
    U.SUITE.check_generate_matches_decode_of_requests("choice", "cpu", F32)


# ---------------------------------------------------------------------------------------------------- the plain statement itself
def _mixer(seed, T=60, H=2, D=8, r=4, E=6, rank=10, W=16, window=11, **kw):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64) / (s[-1] ** 0.5 if len(s) > 1 and s[0] != T else 1.0)
    cfg = U.layer(H, D, r, E, rank, window, None, **kw)["mixer"]
    w = {"q": n(H * (D + r), W), "dkv": n(rank + r, W), "dkv.norm": 1 + 0.1 * n(rank), "uk": n(H * D, rank), "uv": n(H * E, rank), "o": n(W, H * E)}
    return cfg, w, n(T, W)


def test_a_window_shows_its_last_key_and_hides_the_next():
    """Changing the token `window` back changes nothing, changing the one before that edge does."""
    cfg, w, h = _mixer(0)

    def at(i, h):
        c, k = R.latent(w, "", cfg, 1e-5, h)
        return R.latent_attention(w, "", cfg, h, c, k)[i]
    base = at(50, h)
    for gap, seen in ((10, True), (11, False), (0, True), (49, False)):
        h2 = h.clone()
        h2[50 - gap] += 1.0
        assert bool((at(50, h2) - base).abs().max() > 1e-6) == seen, gap


def test_scores_depend_on_distance_only_through_the_rotated_part():
    cfg, w, h = _mixer(1, window=None)
    h = h[:1].expand(40, -1).clone()                         # every token the same: unrotated scores are all equal
    _, k = R.latent(w, "", cfg, 1e-5, h)
    q = R.rotate((h @ w["q"].t()).view(40, 2, 12)[..., 8:], cfg["rot"]["base"])
    s = torch.einsum("ihd,jd->hij", q, k)
    assert torch.allclose(s[:, 30, 25], s[:, 12, 7]) and not torch.allclose(s[:, 30, 25], s[:, 30, 24])


def test_the_correction_takes_part_in_the_choice_but_not_in_the_weights():
    z = torch.tensor([0.0, 1.0, -1.0, 0.5], dtype=torch.float64)
    chosen, weight = R.route(z, torch.zeros(4), 2)
    assert chosen.tolist() == [1, 3]
    chosen, weight = R.route(z, torch.tensor([0.0, -5.0, 5.0, 0.0]), 2)
    assert chosen.tolist() == [2, 3] and torch.allclose(weight, torch.sigmoid(z[[2, 3]]))


# ---------------------------------------------------------------------------------------------------- twins of the kernels
def test_decoding_on_latents_equals_keys_and_values_in_full():
    """The two forms of the same attention, at windows around page and portion edges, with keys that stand out."""
    from litetorch_b200.ops import kernels_ref as K
    g = torch.Generator().manual_seed(0)
    T, H, c, r, d, v = 70, 3, 24, 8, 16, 8
    rows = torch.randn(T, c + r, generator=g)
    uk, uv = torch.randn(H, d, c, generator=g) * c ** -0.5, torch.randn(H, v, c, generator=g) * c ** -0.5
    q = torch.randn(T, H, d + r, generator=g)
    rows[33, c:] = 6 * q[65, 1, d:]                          # 32 back from token 65
    kk, vv = torch.einsum("hdc,tc->thd", uk, rows[:, :c]), torch.einsum("hvc,tc->thv", uv, rows[:, :c])
    table = torch.randperm(9, generator=g)[:5].int()
    cache = torch.full((9, 1, 16, c + r), float("nan"))
    p = torch.arange(T)
    cache[table.long()[p // 16], 0, p % 16] = rows
    for window in (0, 1, 16, 32, 33, 70):
        want = K.shared_rope_fwd(q, kk, rows[:, c:], vv, scale=0.2, window=window)
        ql = torch.cat([torch.einsum("hdc,thd->thc", uk, q[..., :d]), q[..., d:]], 2)
        o = K.latent_decode(ql, cache, table, p.int() + 1, rank=c, window=window, scale=0.2, max_keys=T)
        assert torch.allclose(K.head_linear(o, uv), want, atol=2e-5), window


def test_configurations_that_do_not_fit_are_refused(tmp_path):
    from litetorch_b200.models import registry
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg)
    d = str(tmp_path / "m")
    U.write_model(d, cfg, w)
    assert registry.load_engine(d, "cpu").cfg.vocab == cfg["vocab"]
    with pytest.raises(ValueError, match="l1.mlp.e2.up"):
        U.engine(cfg, dict(w, **{"l1.mlp.e2.up": w["l1.mlp.e2.up"][:, :-1]}), "cpu", F32)
    with pytest.raises(KeyError, match="l3.mlp.correction"):
        U.engine(cfg, {k: t for k, t in w.items() if k != "l3.mlp.correction"}, "cpu", F32)
    assert "l2.mix.dkv" not in w and "l2.norm2" not in w

    def broken(edit):
        c = copy.deepcopy(cfg)
        edit(c["layers"])
        return c
    for edit, words in ((lambda l: l[0].update(type="other"), "unknown type"), (lambda l: l[1]["mlp"].update(kind="other"), "unknown feed-forward"),
                        (lambda l: l[2]["mixer"].update(kv_from=1), "cannot read"), (lambda l: l[2]["mixer"].update(kv_from=2), "cannot read"),
                        (lambda l: l[3]["mixer"].update(kv_from=2), "cannot read"), (lambda l: l[0]["mixer"].update(rot_dim=10), "rotation"),
                        (lambda l: l[1]["mlp"]["router"].update(top=4), "experts")):
        with pytest.raises(ValueError, match=words):
            U.RavenexConfig.parse(broken(edit))
    eng = registry.load_engine(d, "cpu")
    with pytest.raises(ValueError, match="prefix"):
        registry.new_serving(eng, num_blocks=4, prefix_cache_bytes=1 << 20)
    with pytest.raises(TypeError):
        registry.new_serving(eng, num_blocks=4, kv_dtype=torch.bfloat16)


def test_only_layers_with_latents_of_their_own_have_pages():
    cfg = U.CONFIGS["mixed"]
    model, _ = U.server(U.engine(cfg, U.weights(cfg), "cpu", F32))
    assert [t is not None for t in model.cache.k] == [True, True, False, True] and not any(t is not None for t in model.cache.v)
    assert model.cache.bytes_per_token == 4 * sum(t.shape[3] for t in model.cache.k if t is not None)


def test_a_pool_that_is_too_small_refuses_the_session():
    cfg = U.CONFIGS["odd"]
    model, sched = U.server(U.engine(cfg, U.weights(cfg), "cpu", F32), blocks=4, slots=2)
    sched.feed(model, [(1, U.tokens(cfg, 40, 0), [])])
    with pytest.raises(RuntimeError, match="too small"):
        sched.feed(model, [(2, U.tokens(cfg, 40, 0), [])])
    for s in (1, 2):
        sched.end_session(s)
    assert sched.free_blocks == 4


def test_trace_replay(tmp_path):
    from litetorch_b200 import trace
    from litetorch_b200.models import registry
    from litetorch_b200.serving import ServingScheduler
    cfg = U.CONFIGS["choice"]
    w = U.weights(cfg, 8)
    U.write_model(str(tmp_path / "m"), cfg, w)
    a, b = U.tokens(cfg, 50, 1), U.tokens(cfg, 30, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[20:21], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [27, 3]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "b", "tokens": a[:9], "want": [8]}, {"id": "a", "tokens": a[21:], "want": [28]}], "end": ["a", "b"]}]
    said = []
    model = registry.new_serving(registry.load_engine(str(tmp_path / "m"), "cpu"), num_blocks=8, max_num_seqs=2)
    trace.replay(model, ServingScheduler(8, 16, 2, 64), io.StringIO("\n".join(map(json.dumps, steps))), str(tmp_path), said.append)
    assert said == ["done %d" % i for i in range(4)] and not os.path.exists(str(tmp_path / "1.f32"))
    ya, yb = U.SUITE.reference(cfg, w, a), U.SUITE.reference(cfg, w, b)
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


def test_generation_example_and_sampling_on_a_directory(tmp_path):
    cfg = U.CONFIGS["odd"]
    w = U.weights(cfg, 2)
    U.write_model(str(tmp_path / "m"), cfg, w)
    sys.path.insert(0, os.path.join(ROOT, "examples"))
    import generate_llama
    args = ["--model", str(tmp_path / "m"), "--prompt", "5,6,7", "--ids", "--max-new-tokens", "5", "--device", "cpu"]
    seq = [5, 6, 7]
    for t in generate_llama.main(args)["outputs"][0]:
        assert t == int(U.SUITE.reference(cfg, w, seq)[-1].argmax())
        seq.append(t)
    assert len(generate_llama.main(args + ["--temperature", "0.9", "--top-k", "8", "--seed", "3"])["outputs"][0]) == 5


def test_the_engine_loop_of_the_server_runs_the_family():
    from litetorch_b200.models import registry
    from litetorch_b200.server import EngineLoop
    cfg = U.CONFIGS["odd"]
    w = U.weights(cfg, 4)
    model = registry.new_serving(U.engine(cfg, w, "cpu", F32), num_blocks=16, max_num_seqs=2)
    loop = EngineLoop(model, 16, max_num_seqs=2)
    try:
        out = loop.submit([3, 1, 4], 3).generated_tokens
        parts = [t for part in loop.stream([3, 1, 4], 3) for t in part]
    finally:
        loop.close()
    assert out == parts and len(out) == 3
    seq = [3, 1, 4]
    for t in out:
        assert t == int(U.SUITE.reference(cfg, w, seq)[-1].argmax())
        seq.append(t)
