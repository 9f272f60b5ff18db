"""Safuvik on the GPU: every kernel of its mechanisms alone, then prompts, portions, decoding, batches and generation, in
fp32 and bf16, against the plain statement of the equations."""
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import safuvik_ref as R
import safuvik_suite as U

pytestmark = pytest.mark.gpu
F32, BF = torch.float32, torch.bfloat16
DT = [F32, BF]


def _k():
    from litetorch_b200.ops import kernels as K
    return K


def _rand(*shape, dtype=F32, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def _close(got, want, dtype, f32=2e-5, bf16=1.5e-2):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / want.abs().max().clamp(min=1e-3))
    assert err < (f32 if dtype == F32 else bf16), err


def _d(t):
    return t.double().cpu()


# ---------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("streams,width", [(1, 60), (2, 128), (3, 96), (4, 2048), (5, 130), (7, 64)])
def test_streams_and_norm(dtype, streams, width):
    K = _k()
    T, eps = 37, 1e-4
    x = _rand(T, streams, width, seed=1)
    y, y2 = _rand(T, width, dtype=dtype, seed=2), _rand(T, width, dtype=dtype, seed=3)
    n1, n2, norm = _rand(width, seed=4), _rand(width, seed=5), _rand(width, seed=6)
    mix, out, inn = _rand(streams, streams, seed=7), _rand(streams, seed=8), _rand(streams, seed=9)
    for two in (False, True):
        p = {"hc.in": inn.cpu(), "hc.mix": mix.cpu(), "hc.out": out.cpu()}
        add = 0.5 * (R.rms(_d(y), eps, n1.cpu()) + R.rms(_d(y2), eps, n2.cpu())) if two else _d(y)
        want = R.hyper_sublayer(p, "hc.", _d(x), lambda u: add)
        args = dict(y=y, y_norm=n1, y2=y2, y2_norm=n2) if two else dict(y=y)
        rows = torch.tensor([36, 0, 5], dtype=torch.int32, device="cuda")
        xs = x.clone()
        h = K.hyper_norm(xs, norm, eps, dtype=dtype, rows=rows, write=False, mix=mix, out=out, **args)
        _close(h, R.rms(want.sum(1), eps, norm.cpu())[[36, 0, 5]], dtype)
        assert torch.equal(xs, x)
        h = K.hyper_norm(xs, norm, eps, dtype=dtype, inn=inn, mix=mix, out=out, **args)
        _close(xs, want, F32)
        _close(h, R.rms(torch.einsum("s,tsw->tw", _d(inn), want), eps, norm.cpu()), dtype)
    table, tok = _rand(11, width, dtype=dtype, seed=10), torch.tensor([3, 10, 0, 7], dtype=torch.int32, device="cuda")
    xs = torch.full((4, streams, width), math.nan, device="cuda")
    h = K.hyper_norm(xs, norm, eps, dtype=dtype, inn=inn, tokens=tok, embed=table)
    e = _d(table)[tok.long().cpu()]
    _close(xs, e[:, None].expand(4, streams, width), F32)
    _close(h, R.rms(e * float(inn.double().sum()), eps, norm.cpu()), dtype, f32=1e-4)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,G,D,E,dims", [(4, 2, 24, 40, 12), (8, 1, 128, 64, 128), (5, 5, 10, 6, 0), (2, 1, 144, 160, 100)])
def test_projection_norm_and_rotation(dtype, H, G, D, E, dims):
    K = _k()
    N, bs, eps = 9, 16, 1e-5
    rot = {"base": 900.0, "dims": dims, "scaling": {"factor": 6.0, "original": 512, "fast": 16.0, "slow": 1.0}}
    freq, gain = R.inverse_frequencies(rot) if dims else (torch.zeros(1, dtype=torch.float64), 1.0)
    r8 = lambda n: (n + 7) // 8 * 8
    DP, EP = r8(D) + 8, r8(E)
    offs = [8, 8 + r8(H * D), 8 + r8(H * D) + r8(G * D)]
    proj = _rand(N, offs[2] + r8(G * E), dtype=dtype, seed=1)
    qn, kn = _rand(H * D, seed=2), _rand(G * D, seed=3)
    pos = torch.tensor([0, 1, 2, 63, 64, 65, 4095, 70001, 1000003], dtype=torch.int32)
    slots = torch.tensor([5, 16, 31, 32, 47, 0, 100, 63, 64], dtype=torch.int32)
    kc, vc = torch.full((8, G, bs, DP), 7.0, dtype=dtype, device="cuda"), torch.full((8, G, bs, EP), 7.0, dtype=dtype, device="cuda")
    lin = torch.empty(N, G, DP, dtype=dtype, device="cuda"), torch.empty(N, G, EP, dtype=dtype, device="cuda")
    q = K.qkv_rope(proj, *offs, H, G, D, E, pos.cuda(), slots.cuda(), kc, vc, freq=freq.cuda(), rot_dims=dims, gain=gain, q_norm=qn, k_norm=kn,
                   eps=eps, lin=lin)

    def want(off, heads, w):
        t = R.rms(_d(proj)[:, off:off + heads * D], eps, w.cpu()).view(N, heads, D)
        a = pos.double()[:, None] * freq[None]
        y = t.clone()
        if dims:
            c, s = (torch.cos(a) * gain)[:, None], (torch.sin(a) * gain)[:, None]
            y[..., 0:dims:2] = t[..., 0:dims:2] * c - t[..., 1:dims:2] * s
            y[..., 1:dims:2] = t[..., 1:dims:2] * c + t[..., 0:dims:2] * s
        return y
    _close(q[..., :D], want(offs[0], H, qn), dtype)
    _close(lin[0][..., :D], want(offs[1], G, kn), dtype)
    assert torch.equal(lin[1][..., :E].reshape(N, -1), proj[:, offs[2]:offs[2] + G * E])
    for t in (q[..., D:], lin[0][..., D:], lin[1][..., E:]):
        assert not bool(t.any())
    blk, off = slots.long() // bs, slots.long() % bs
    assert torch.equal(kc[blk, :, off], lin[0]) and torch.equal(vc[blk, :, off], lin[1])
    kc[blk, :, off] = 7.0
    assert bool((kc == 7.0).all())                            # nothing but the given cells was written


def _paged(k, v, DP, EP, dtype, seed=0):
    """Keys and values [T, G, .] in shuffled blocks of 16."""
    T, G, _ = k.shape
    nb = (T + 15) // 16
    table = torch.randperm(nb + 3, generator=torch.Generator().manual_seed(seed))[:nb]
    kc = torch.full((nb + 3, G, 16, DP), math.nan, dtype=dtype)
    vc = torch.full((nb + 3, G, 16, EP), math.nan, dtype=dtype)
    kc[table], vc[table] = 0.0, 0.0
    p = torch.arange(T)
    kc[table[p // 16], :, p % 16] = torch.nn.functional.pad(k, (0, DP - k.shape[2])).to(dtype)
    vc[table[p // 16], :, p % 16] = torch.nn.functional.pad(v, (0, EP - v.shape[2])).to(dtype)
    return kc.cuda(), vc.cuda(), table.int().cuda()


def _edge_case(T, H, G, D, E, window, dtype, seed=0):
    """q, k, v in which, for many queries, one key just inside or just outside the window would take all the weight."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(T, n, m, generator=g) for n, m in ((H, D), (G, D), (G, E)))
    for n, t in enumerate(range(T - 1, 0, -3)):
        gap = (window - 1, window, window + 1, 0, 1)[n % 5]
        if t - gap >= 0:
            k[t - gap] = q[t].view(G, H // G, D)[:, -1] * 3.0
    return tuple(t.to(dtype) for t in (q, k, v))


@pytest.mark.parametrize("window", [1, 2, 17, 127, 128, 129, 256, 300, 5000])
@pytest.mark.parametrize("D", [64, 128])
def test_window_in_the_prompt_kernel(D, window):
    K = _k()
    H, G = 4, 2
    for Tk, Tq in ((400, 400), (129, 129), (333, 70), (700, 300), (50, 2), (257, 1)):
        q, k, v = _edge_case(Tk, H, G, D, D, window, BF, seed=Tk)
        want = R.window_attention(q.double(), k.double(), v.double(), D ** -0.5, window)[Tk - Tq:]
        o, _ = K.flash_fwd(q[Tk - Tq:].cuda()[None], k.cuda()[None], v.cuda()[None], causal=True, scale=D ** -0.5, window=window)
        _close(o[0], want, BF, bf16=2e-2)
    assert K.status_fetch() == 0


def test_window_rows_that_see_very_low_scores_only():
    """A row whose visible keys all score far below zero, after whole tiles that it does not see."""
    K = _k()
    T, D, window = 512, 64, 20
    q = torch.zeros(T, 1, D)
    k = torch.zeros(T, 1, D)
    q[:, :, 0] = 30.0
    k[:, :, 0] = -30.0 - torch.arange(T)[:, None] * 0.01
    v = torch.randn(T, 1, D, generator=torch.Generator().manual_seed(0))
    q, k, v = q.to(BF), k.to(BF), v.to(BF)
    want = R.window_attention(q.double(), k.double(), v.double(), 1.0, window)
    o, _ = K.flash_fwd(q.cuda()[None], k.cuda()[None], v.cuda()[None], causal=True, scale=1.0, window=window)
    _close(o[0], want, BF, bf16=2e-2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,G,D,E,window", [(4, 2, 24, 40, 37), (8, 1, 128, 64, 129), (17, 1, 10, 6, 16), (2, 1, 144, 160, 50), (20, 1, 64, 64, 33),
                                            (4, 4, 64, 64, 1), (6, 3, 128, 128, 160)])
def test_window_in_decoding_and_on_the_cuda_cores(dtype, H, G, D, E, window):
    K = _k()
    T = 230
    q, k, v = _edge_case(T, H, G, D, E, window, dtype, seed=H)
    gate = _rand(T, H + 3, dtype=dtype, seed=5)[:, 3:]
    want = R.window_attention(q.double(), k.double(), v.double(), 0.2, window) * torch.sigmoid(_d(gate))[..., None]
    r8 = lambda n: (n + 7) // 8 * 8
    kc, vc, table = _paged(k, v, r8(D), r8(E), dtype)
    qp = torch.nn.functional.pad(q, (0, r8(D) - D)).cuda()
    pos = torch.arange(T, dtype=torch.int32).cuda()
    o = K.window_attn(qp, kc, vc, table, pos, D=D, E=E, window=window, scale=0.2, gate=gate)
    _close(o, want, dtype, bf16=2e-2)
    rows = [0, 1, 15, 16, 17, 36, 37, 38, 128, 129, 130, 159, 160, 161, 229]          # as one token of many sequences
    tables = table[None].repeat(len(rows), 1).contiguous()
    o = K.window_attn(qp[rows].contiguous(), kc, vc, tables, pos[rows].contiguous(), D=D, E=E, window=window, scale=0.2, gate=gate[rows])
    _close(o, want[rows], dtype, bf16=2e-2)
    if dtype == BF and max(D, E) <= 128:
        P = 64 if max(D, E) <= 64 else 128
        kc, vc, table = _paged(k, v, P, P, dtype, seed=1)
        tables = table[None].repeat(len(rows), 1).contiguous()
        qp = torch.nn.functional.pad(q[rows], (0, P - D)).cuda()
        for splits in (1, 2, 5):
            o = K.paged_decode(qp, kc, vc, tables, pos[rows] + 1, 16, splits, 0.2, window=window, gate=gate[rows], vdim=E)
            _close(o, want[rows], dtype, bf16=2e-2)
        lin = torch.empty(2, 40, G, P, dtype=dtype, device="cuda")
        K.kv_gather(kc, vc, table, 101, 40, lin[0], lin[1])
        assert torch.equal(lin[0, ..., :D].cpu(), k[101:141]) and torch.equal(lin[1, ..., :E].cpu(), v[101:141])
    _close(K.head_gate(_pad_v(v, H, G, r8(E)), gate, E), v.double().repeat_interleave(H // G, 1) * torch.sigmoid(_d(gate))[..., None], dtype)
    assert K.status_fetch() == 0


def _pad_v(v, H, G, EP):
    return torch.nn.functional.pad(v.repeat_interleave(H // G, 1), (0, EP - v.shape[2])).contiguous().cuda()


def _recurrence(C, blocks, taps, T, dtype, seed=0):
    bw = C // blocks
    f = lambda *s, k, scale=1.0: _rand(*s, seed=seed + k, scale=scale)
    w = dict(x=_rand(T, C + 8, dtype=dtype, seed=seed)[:, 8:], y=_rand(T, 2 * C, dtype=dtype, seed=seed + 1)[:, :C], xb=f(C, k=2), yb=f(C, k=3),
             conv=f(C, taps, k=4), conv_b=f(C, k=5), gates=_rand(blocks, 2 * bw, bw, dtype=dtype, seed=seed + 6, scale=bw ** -0.5),
             rb=f(blocks, bw, k=7), ib=f(blocks, bw, k=8), lam=f(C, k=9) - 2.0)
    w["sp"] = torch.nn.functional.softplus(w["lam"].double()).float()
    u = R.causal_conv(_d(w["x"]) + _d(w["xb"]), _d(w["conv"]), w["conv_b"].cpu())
    if dtype == BF:
        u = u.to(BF).double()
    r = torch.sigmoid(R.block_diagonal(u, w["gates"][:, :bw].cpu(), w["rb"].cpu()))
    i = torch.sigmoid(R.block_diagonal(u, w["gates"][:, bw:].cpu(), w["ib"].cpu()))
    s = R.gated_linear_recurrence(u, r, i, w["lam"].cpu())
    return w, u, s, s * R.gelu(_d(w["y"]) + _d(w["yb"]))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("C,blocks,taps", [(80, 5, 3), (256, 2, 4), (256, 4, 4), (33, 3, 1), (64, 1, 6), (512, 2, 2)])
def test_convolution_and_recurrence(dtype, C, blocks, taps):
    K = _k()
    T = 300
    w, u, s, want = _recurrence(C, blocks, taps, T, dtype)
    state, ring = torch.full((3, C), math.nan, device="cuda"), torch.full((3, taps, C), math.nan, device="cuda")

    def prompt(a, b, slot):
        x, y = w["x"][a:b], w["y"][a:b]
        uu = K.conv_causal(x, w["xb"], w["conv"], w["conv_b"], ring[slot], a)
        _close(uu, u[a:b], dtype)
        return K.rglru_scan(uu, K.block_diag(uu, w["gates"]), w["rb"], w["ib"], w["sp"], y, w["yb"], x, w["xb"], state[slot], ring[slot], taps, a)

    cuts = [0, 130, 132, 133, 134, 262, 297]
    for a, b in zip(cuts, cuts[1:]):
        _close(prompt(a, b, 1), want[a:b], dtype, bf16=2.5e-2)
    _close(state[1], s[296], dtype, bf16=2.5e-2)
    _close(prompt(0, 297, 2), want[:297], dtype, bf16=2.5e-2)
    # single steps of two sequences that stand at different places, one from its very first token
    slots = torch.tensor([2, 0], dtype=torch.int32, device="cuda")
    for k in range(3):
        rows = [297 + k, k]
        pos = torch.tensor(rows, dtype=torch.int32, device="cuda")
        o = K.rglru_step(w["x"][rows], w["xb"], w["conv"], w["conv_b"], w["gates"], w["rb"], w["ib"], w["sp"], w["y"][rows], w["yb"], state, ring,
                         slots, pos)
        _close(o, want[rows], dtype, bf16=2.5e-2)
    assert torch.equal(state[1], state[1]) and K.status_fetch() == 0


@pytest.mark.parametrize("dtype", DT)
def test_recurrence_steps_of_many_sequences(dtype):
    K = _k()
    C, blocks, taps, n = 256, 2, 4, 37                           # more sequences than one CTA takes
    w, _, _, want = _recurrence(C, blocks, taps, n, dtype)
    state, ring = torch.zeros(n + 1, C, device="cuda"), torch.zeros(n + 1, taps, C, device="cuda")
    for t in range(5):
        slots = torch.arange(n - 1, -1, -1, dtype=torch.int32, device="cuda")
        pos = torch.full((n,), t, dtype=torch.int32, device="cuda")
        rows = [t] * n
        o = K.rglru_step(w["x"][rows], w["xb"], w["conv"], w["conv_b"], w["gates"], w["rb"], w["ib"], w["sp"], w["y"][rows], w["yb"], state, ring,
                         slots, pos)
        _close(o, want[rows], dtype, bf16=2.5e-2)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,D,E,forget,gain", [(3, 20, 28, 3.0, 1.0), (2, 64, 128, 3.0, 1.0), (1, 7, 5, 0.0, 1.0), (2, 70, 66, -4.0, 2.0), (2, 130, 132, 6.0, 6.0),
                                               (2, 128, 256, 5.0, 1.0)])
def test_matrix_memory(dtype, H, D, E, forget, gain):
    K = _k()
    T, cap, eps = 420, 8.0, 1e-5
    r8 = lambda n: (n + 7) // 8 * 8
    offs = [0, r8(H * D), 2 * r8(H * D), 2 * r8(H * D) + r8(H * E)]
    proj = _rand(T, offs[3] + r8(H * E), dtype=dtype, seed=1)
    cut = lambda rows: (proj[rows, offs[0]:offs[0] + H * D], proj[rows, offs[1]:offs[1] + H * D], proj[rows, offs[2]:offs[2] + H * E],
                        proj[rows, offs[3]:offs[3] + H * E])
    logits = _rand(T, 2 * H, seed=2) * gain
    ib, fb, norm = _rand(H, seed=3), _rand(H, seed=4) + forget, _rand(H * E, seed=5)
    i = cap * torch.tanh(_d(logits[:, :H] + ib) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(_d(logits[:, H:] + fb) / cap))
    q, k, v, gate = (_d(t) for t in cut(slice(None)))
    o = R.matrix_memory(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, E), i, f)
    want = R.rms(o, eps).reshape(T, H * E) * _d(norm) * torch.sigmoid(gate)
    nan = lambda *s: torch.full(s, math.nan, device="cuda")
    S, n, m = nan(3, H, D, E), nan(3, 2, H, D), nan(3, 2, H)

    def prompt(a, b, slot):
        q, k, v, gate = cut(slice(a, b))
        return K.mlstm_prefill(q, k, v, logits[a:b].contiguous(), ib, fb, cap, norm, eps, gate, S[slot], n[slot], m[slot], D, E, a)

    tol = dict(f32=3e-4, bf16=2e-2)                 # a head whose output nearly cancels is blown up by its norm
    cuts = [0, 128, 130, 131, 259, 387, 417]
    for a, b in zip(cuts, cuts[1:]):
        _close(prompt(a, b, 1), want[a:b], dtype, **tol)
    _close(prompt(0, 417, 2), want[:417], dtype, **tol)
    slots = torch.tensor([1, 0], dtype=torch.int32, device="cuda")
    for t in range(3):
        rows = [417 + t, t]
        qq, kk, vv, gg = (x.contiguous() for x in cut(rows))
        y = K.mlstm_step(*(proj[rows][:, o:o + w] for o, w in zip(offs[:3], (H * D, H * D, H * E))), logits[rows], ib, fb, cap, norm, eps, gg, S, n, m,
                         slots, torch.tensor(rows, dtype=torch.int32, device="cuda"), D, E)
        _close(y, want[rows], dtype, **tol)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("M,F,limit", [(5, 35, 0.5), (300, 1024, 7.0), (1, 8, 1.0)])
def test_clamped_feed_forward_unit(dtype, M, F, limit):
    gu = _rand(M, 2 * F, dtype=dtype, scale=2.0 * limit)
    _close(_k().clamped_glu(gu, limit), R.clamped_glu(_d(gu)[:, :F], _d(gu)[:, F:], limit), dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("M,N,Kd", [(1, 77, 60), (9, 35, 60), (130, 131, 33), (64, 64, 64), (5, 1024, 256), (200, 999, 520)])
def test_products(dtype, M, N, Kd):
    K = _k()
    x, w = _rand(M, Kd, dtype=dtype), _rand(N, Kd, dtype=dtype, seed=1)
    want = _d(x) @ _d(w).t()
    _close(K.linear(x, w), want, dtype)
    _close(K.linear(x, w, out_dtype=F32, alpha=0.3), 0.3 * want, F32)
    _close(K.rows_dot(x, w[:20].contiguous()), want[:, :20], F32)
    b = _rand(3, 2 * 64, 40, dtype=dtype, seed=2)
    xb = _rand(M, 120, dtype=dtype, seed=3)
    _close(K.block_diag(xb, b), torch.cat([_d(xb)[:, 40 * z:40 * z + 40] @ _d(b)[z].t() for z in range(3)], 1), F32)


# ---------------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_portions_of_all_sizes(name, dtype):
    U.check_portions(name, "cuda", dtype, 300, [[300], [250, 1], [2], [64, 3], [127, 2, 1, 1, 1, 126, 1], [129, 128, 1], [5, 17, 2, 37]])
    assert _k().status_fetch() == 0


@pytest.mark.parametrize("dtype", DT)
def test_long_decoding_from_the_first_token(dtype):
    U.check_portions("tiles", "cuda", dtype, 420, [[1]])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_requests_side_by_side_and_reused_pages_and_slots(name, dtype):
    U.check_interleaved(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(name, dtype):
    U.check_generate(name, "cuda", dtype, 20, 16)


def test_requests_that_share_a_batch_do_not_see_each_other():
    U.check_generate_matches_decode_of_requests("cuda", F32)


def test_graph_replay_and_eager_decoding_agree():
    """The pass that records a decode step must not advance the recurrent state."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg)
    from litetorch_b200.models import registry
    eng = U.engine(cfg, w, "cuda", BF)
    toks = U.tokens(cfg, 40, 2)
    outs = []
    for graphs in (False, True):
        model = registry.new_serving(eng, num_blocks=8, max_num_seqs=2, graphs=graphs)
        _, sched = None, U.ServingScheduler(8, 16, 2, 4096, -1)
        outs.append(U.run_portions(model, sched, 0, toks, [10, 1]))
    assert float((outs[0] - outs[1]).abs().max()) < 1e-3
