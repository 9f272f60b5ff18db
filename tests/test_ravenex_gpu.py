"""Ravenex on the GPU: every kernel of its mechanisms alone, then prompts, portions, decoding, batches and generation, in
fp32 and bf16, against the plain statement of the equations."""
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ravenex_ref as R
import ravenex_suite as U

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
@pytest.mark.parametrize("T,W", [(37, 60), (5, 2048), (600, 96), (400, 4096), (3, 7777), (2, 1), (300, 333), (1, 12288)])
def test_residual_and_norms(dtype, T, W):
    K = _k()
    eps, m = 1e-3, 0.6
    x, y, wb, wn = _rand(T, W, seed=1), _rand(T, W + 4, dtype=dtype, seed=2)[:, :W], _rand(W, seed=3), _rand(W, seed=4)
    want = _d(x) + m * R.rms(_d(y), eps, wb.cpu())
    rows = torch.tensor([T - 1, 0], dtype=torch.int32, device="cuda")
    xs = x.clone()
    h = K.residual_norm(xs, eps, dtype=dtype, norm=wn, mult=m, y=y, y_norm=wb, rows=rows, write=False)
    _close(h, R.rms(want, eps, wn.cpu())[[T - 1, 0]], dtype)
    assert torch.equal(xs, x)
    h = K.residual_norm(xs, eps, dtype=dtype, norm=wn, mult=m, y=y, y_norm=wb)
    _close(xs, want, F32)
    _close(h, R.rms(want, eps, wn.cpu()), dtype)
    # the residual itself instead of its norm, and an output that is not normed
    xs = x.clone()
    h = K.residual_norm(xs, eps, dtype=dtype, mult=m, y=y)
    _close(xs, _d(x) + m * _d(y), F32)
    _close(h, _d(x) + m * _d(y), dtype)
    # a weighted sum of rows elsewhere, alone and on top of y
    z, top = _rand(T * 3 + 5, W, dtype=dtype, seed=5), 3
    slots = torch.randperm(T * 3 + 5, generator=torch.Generator().manual_seed(T))[:T * top].view(T, top).int().cuda()
    a = _rand(T, top, seed=6)
    s = (_d(z)[slots.long().cpu()] * _d(a)[..., None]).sum(1)
    for base in (None, y):
        xs = x.clone()
        h = K.residual_norm(xs, eps, dtype=dtype, norm=wn, mult=m, y=base, y_norm=wb, experts=(z, slots, a))
        want = _d(x) + m * R.rms(s if base is None else s + _d(base), eps, wb.cpu())
        _close(xs, want, F32, f32=5e-5)
        _close(h, R.rms(want, eps, wn.cpu()), dtype, f32=5e-5)
    # the start of the residual
    table, tok = _rand(11, W, dtype=dtype, seed=10), torch.tensor([3, 10, 0, 7], dtype=torch.int32, device="cuda")
    xs = torch.full((4, W), math.nan, device="cuda")
    h = K.residual_norm(xs, eps, dtype=dtype, norm=wn, mult=m, tokens=tok, embed=table)
    e = _d(table)[tok.long().cpu()]
    assert torch.equal(xs.double().cpu(), e)
    _close(h, R.rms(e, eps, wn.cpu()), dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,d,r,rot,rank,c", [(3, 24, 16, 12, 40, 40), (16, 128, 64, 64, 512, 512), (1, 8, 8, 2, 21, 64), (5, 64, 64, 32, 130, 192), (2, 16, 104, 104, 7, 8)])
@pytest.mark.parametrize("in_place", [True, False])
def test_rotation_latent_norm_and_cache_write(dtype, H, d, r, rot, rank, c, in_place):
    K = _k()
    N, bs, eps, base = 9, 16, 1e-4, 900.0
    q_cols = H * (d + r)
    proj = _rand(N, q_cols + rank + rot + (-(q_cols + rank + rot)) % 64, dtype=dtype, seed=1)
    wc = _rand(rank, seed=3)
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    pos = torch.tensor([0, 1, 2, 63, 64, 65, 4095, 70001, 1000003], dtype=torch.int32)
    slots = torch.tensor([5, 16, 31, 32, 47, 0, 100, 63, 64], dtype=torch.int32)
    cache = torch.full((8, 1, bs, c + r), 7.0, dtype=dtype, device="cuda")
    lin = torch.empty(N, c + r, dtype=dtype, device="cuda")
    before = proj.clone()
    q_out = None if in_place else torch.full((N, H, c + r), 3.0, dtype=dtype, device="cuda")
    K.latent_rope(proj, H, d, r, rot, pos.cuda(), slots.cuda(), freq=freq.cuda(), c_off=q_cols, rank=rank, c_norm=wc, eps=eps, cache=cache,
                  q_out=q_out, lin=lin)

    def turn(x):
        a = pos.double()[:, None] * freq
        a = a if x.dim() == 2 else a[:, None]
        u, v = x[..., 0::2], x[..., 1::2]
        return torch.stack([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)], -1).flatten(-2)
    heads = _d(before)[:, :q_cols].view(N, H, d + r)
    got = proj[:, :q_cols].view(N, H, d + r)[..., d:] if in_place else q_out[..., c:]
    _close(got[..., :rot], turn(heads[..., d:d + rot]), dtype)
    assert not bool(got[..., rot:].any())
    if in_place:
        assert torch.equal(proj[:, :q_cols].view(N, H, d + r)[..., :d], before[:, :q_cols].view(N, H, d + r)[..., :d])
    else:
        assert torch.equal(proj, before) and bool((q_out[..., :c] == 3.0).all())
    _close(lin[:, :rank], R.rms(_d(before)[:, q_cols:q_cols + rank], eps, wc.cpu()), dtype)
    _close(lin[:, c:c + rot], turn(_d(before)[:, q_cols + rank:q_cols + rank + rot]), dtype)
    assert not bool(lin[:, rank:c].any()) and not bool(lin[:, c + rot:].any())
    blk, off = slots.long() // bs, slots.long() % bs
    assert torch.equal(cache[blk, 0, off], lin)
    cache[blk, 0, off] = 7.0
    assert bool((cache == 7.0).all())                         # nothing but the given cells was written
    # a layer without latents of its own rotates its queries alone
    alone = before.clone()
    K.latent_rope(alone, H, d, r, rot, pos.cuda(), slots.cuda(), freq=freq.cuda())
    _close(alone[:, :q_cols].view(N, H, d + r)[..., d:d + rot], turn(heads[..., d:d + rot]), dtype)
    assert torch.equal(alone[:, q_cols:], before[:, q_cols:])


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("N,H,Kd,M", [(1, 1, 64, 64), (7, 3, 128, 512), (33, 16, 512, 128), (300, 2, 64, 128), (5, 4, 24, 21), (130, 3, 96, 8)])
def test_product_per_head(dtype, N, H, Kd, M):
    K = _k()
    x, w = _rand(N, H, Kd + 16, dtype=dtype, seed=1)[..., 8:8 + Kd], _rand(H, M, Kd, dtype=dtype, seed=2)
    want = torch.einsum("nhk,hmk->nhm", _d(x), _d(w))
    _close(K.head_linear(x, w), want, dtype)
    big = torch.full((N, H, M + 24), 5.0, dtype=dtype, device="cuda")
    K.head_linear(x, w, out=big[..., 8:8 + M])
    _close(big[..., 8:8 + M], want, dtype)
    assert bool((big[..., :8] == 5.0).all()) and bool((big[..., 8 + M:] == 5.0).all())


def _edge_rows(T, H, d, v, window, seed):
    """Queries, unrotated keys, shared key part and values in which, for many queries, one key just inside or just outside the
    window would take all the weight - through the part that all heads share."""
    g = torch.Generator().manual_seed(seed)
    q, k, ks, vv = (torch.randn(*s, generator=g) for s in ((T, H, d + 64), (T, H, d), (T, 64), (T, H, v)))
    for n, t in enumerate(range(T - 1, 0, -3)):
        gap = (window - 1, window, window + 1, 0, 1)[n % 5] if window else (t, 0, t // 2)[n % 3]
        if t - gap >= 0:
            ks[t - gap] = q[t, n % H, d:] * 3.0
    return tuple(t.to(BF) for t in (q, k, ks, vv))


@pytest.mark.parametrize("window", [0, 1, 2, 17, 63, 64, 65, 127, 128, 129, 300, 5000])
@pytest.mark.parametrize("d,v", [(64, 64), (64, 128), (128, 128)])
def test_prompt_attention_with_a_shared_key_part(d, v, window):
    K = _k()
    H = 3
    for Tk, Tq in ((400, 400), (129, 129), (333, 70), (700, 300), (50, 2), (257, 1), (64, 64)):
        q, k, ks, vv = _edge_rows(Tk, H, d, v, window, seed=Tk)
        score = torch.einsum("ihd,jhd->hij", q[..., :d].double(), k.double()) + torch.einsum("ihd,jd->hij", q[..., d:].double(), ks.double())
        want = torch.einsum("hij,jhe->ihe", R.windowed_softmax(score * 0.11, window or None), vv.double())[Tk - Tq:]
        # operands as columns of wider rows
        kv = torch.cat([k.reshape(Tk, -1), vv.reshape(Tk, -1)], 1).cuda()
        rows = torch.cat([torch.randn(Tk, 64).to(BF), ks], 1).cuda()
        qq = torch.cat([q.reshape(Tk, -1), torch.zeros(Tk, 64, dtype=BF)], 1).cuda()[Tk - Tq:]
        o = K.shared_rope_fwd(qq[:, :H * (d + 64)].unflatten(1, (H, d + 64)), kv[:, :H * d].unflatten(1, (H, d)), rows[:, 64:],
                              kv[:, H * d:].unflatten(1, (H, v)), scale=0.11, window=window)
        _close(o, want, BF, bf16=2e-2)
    assert K.status_fetch() == 0


def _paged_rows(T, w, seed, block_size=16):
    g = torch.Generator().manual_seed(seed)
    rows = torch.randn(T, w, generator=g).to(BF)
    nb = (T + block_size - 1) // block_size
    table = torch.randperm(nb + 3, generator=g)[:nb].int()
    cache = torch.full((nb + 3, 1, block_size, w), math.nan, dtype=BF)      # rows past the sequence are never read
    p = torch.arange(T)
    cache[table.long()[p // block_size], 0, p % block_size] = rows
    return rows, cache, table


@pytest.mark.parametrize("c,r", [(64, 64), (128, 64), (320, 64), (512, 64)])
@pytest.mark.parametrize("H", [1, 4, 16, 17, 32, 40])
def test_decode_attention_on_latents(c, r, H):
    K = _k()
    w = c + r
    ctxs = [1, 2, 15, 16, 17, 63, 64, 65, 128, 300, 777]
    for window, splits, bs in ((0, 1, 16), (0, 0, 16), (37, 0, 16), (64, 2, 8), (65, 3, 32), (300, 5, 16), (1, 1, 16)):
        caches, tables, rows, qs = [], [], [], []
        at = 0
        for n, T in enumerate(ctxs):
            row, cache, table = _paged_rows(T, w, 100 * n + c + H, bs)
            q = torch.randn(H, w, generator=torch.Generator().manual_seed(n)).to(BF)
            gap = (window - 1, window, 0)[n % 3] if window else (0, T - 1, T // 2)[n % 3]      # one row that stands out, at an edge
            if 0 <= T - 1 - gap:
                row[T - 1 - gap] = (q[n % H].float() * 2.0).to(BF)
                cache[int(table[(T - 1 - gap) // bs]), 0, (T - 1 - gap) % bs] = row[T - 1 - gap]
            caches.append(cache)
            tables.append(table + at)
            rows.append(row)
            qs.append(q)
            at += cache.shape[0]
        width = max(len(t) for t in tables)
        tab = torch.zeros(len(ctxs), width, dtype=torch.int32)
        for i, t in enumerate(tables):
            tab[i, :len(t)] = t
        o = K.latent_decode(torch.stack(qs).cuda(), torch.cat(caches).cuda(), tab.cuda(), torch.tensor(ctxs, dtype=torch.int32, device="cuda"), rank=c,
                            window=window, scale=0.07, max_keys=min(window, 777) if window else 777, splits=splits)
        for i, T in enumerate(ctxs):
            seen = rows[i][max(0, T - window) if window else 0:].double()
            a = torch.softmax(qs[i].double() @ seen.t() * 0.07, -1)
            _close(o[i], a @ seen[:, :c], BF, bf16=1.5e-2)
    assert K.status_fetch() == 0


@pytest.mark.parametrize("N,E,top", [(1, 8, 3), (5, 1, 1), (64, 64, 6), (64, 33, 33), (65, 8, 3), (500, 64, 6), (300, 200, 8), (1000, 7, 2), (17, 1000, 16)])
def test_choice_of_experts_and_their_slots(N, E, top):
    K = _k()
    z = _rand(N, E, seed=N) * 2
    corr = _rand(E, seed=1) * 0.7
    corr[E // 2] += 0.5                                       # a popular expert
    if N > 2:
        z[2] = 0.25                                           # ties: the first experts win
    for br in (16, 64, 128):
        x = _rand(N, 40, dtype=BF, seed=3) if N > 64 else None
        p = K.moe_plan(z, corr, top, br, x)
        slot, group, rows, live = p["slot"].cpu().long(), p["group"].cpu(), p["rows"].cpu(), int(p["live"])
        assert live <= p["blocks"] and slot.unique().numel() == N * top and int(slot.max()) < live * br
        expert = group[slot // br].long()
        s = torch.sigmoid(_d(z))
        for n in range(N):
            chosen, weight = R.route(_d(z)[n], corr.cpu(), top)
            if not torch.equal(chosen, expert[n]):            # a tie up to fp32 rounding: the same choice scores all the same
                cs = s[n] + _d(corr)
                assert torch.allclose(cs[chosen], cs[expert[n]], atol=1e-6), n
            assert torch.allclose(_d(p["weight"])[n], s[n][expert[n]], atol=1e-6)
        used = torch.zeros(live, dtype=torch.long).index_add_(0, slot.reshape(-1) // br, torch.ones(N * top, dtype=torch.long))
        assert torch.equal(used, rows[:live].long())
        assert bool((slot % br < rows[slot // br]).all())
        tok = torch.arange(N).repeat_interleave(top)
        assert torch.equal(p["src"].cpu().long()[slot.reshape(-1)], tok)
        if x is not None:
            assert torch.equal(p["xs"].cpu()[slot.reshape(-1)], x.cpu()[tok])


def test_tied_experts_are_taken_in_order():
    K = _k()
    for E in (6, 70):
        z = torch.full((70, E), 0.5, device="cuda")
        for n in (3, 70):
            p = K.moe_plan(z[:n].contiguous(), torch.zeros(E, device="cuda"), 4, 16)
            e = p["group"].cpu()[p["slot"].cpu().long() // 16]
            assert torch.equal(e, torch.arange(4).int().expand(n, 4))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("N,E,top,W,F", [(1, 8, 3, 64, 32), (32, 64, 6, 256, 96), (64, 4, 2, 96, 64), (64, 2, 2, 64, 32), (200, 40, 2, 64, 64),
                                         (200, 8, 3, 128, 160), (700, 5, 4, 264, 96), (130, 6, 2, 60, 32), (9, 5, 1, 50, 64)])
def test_experts(dtype, N, E, top, W, F):
    K = _k()
    x = _rand(N, W, dtype=dtype, seed=1)
    gu, down = _rand(E, 2 * F, W, dtype=dtype, seed=2, scale=W ** -0.5), _rand(E, W, F, dtype=dtype, seed=3, scale=F ** -0.5)
    router, corr = _rand(E, W, dtype=dtype, seed=4, scale=2 * W ** -0.5), _rand(E, seed=5)
    z, slot, weight = K.moe_experts(x, router, corr, top, gu, down, "silu")
    logits = _d(x) @ _d(router).t()
    s = torch.sigmoid(logits)
    best = torch.argsort(s + _d(corr), dim=1, descending=True)[:, :top]
    assert torch.allclose(_d(weight), s.gather(1, best), atol=1e-5)          # random reals: no close calls here
    rows = z.double().cpu()[slot.long().cpu()]
    want = torch.empty(N, top, W, dtype=torch.float64)
    for e in range(E):
        n, j = (best == e).nonzero(as_tuple=True)
        h = R.silu(_d(x)[n] @ _d(gu)[e, :F].t()) * (_d(x)[n] @ _d(gu)[e, F:].t())
        want[n, j] = h @ _d(down)[e].t()
    _close(rows, want, dtype)
    assert K.status_fetch() == 0


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("act", ["gelu", "silu"])
@pytest.mark.parametrize("M,W,F", [(1, 64, 32), (16, 256, 96), (17, 2048, 512), (70, 128, 40), (128, 64, 64), (300, 96, 72), (5, 50, 35)])
def test_gated_feed_forward(dtype, act, M, W, F):
    K = _k()
    x = _rand(M, W, dtype=dtype, seed=1)
    gu, down = _rand(2 * F, W, dtype=dtype, seed=2, scale=2 * W ** -0.5), _rand(W, F, dtype=dtype, seed=3, scale=F ** -0.5)
    f = R.gelu if act == "gelu" else R.silu
    h = f(_d(x) @ _d(gu)[:F].t()) * (_d(x) @ _d(gu)[F:].t())
    _close(K.glu_mlp(x, gu, down, act), h @ _d(down).t(), dtype)
    big = _rand(M, 2 * F, dtype=dtype, seed=4, scale=3.0)
    _close(K.act_glu(big, act), f(_d(big)[:, :F]) * _d(big)[:, F:], dtype)


@pytest.mark.parametrize("M,N,Kd", [(129, 8, 64), (300, 72, 40), (128, 256, 512), (1000, 1000, 264), (257, 2056, 2048), (40, 64, 8)])
def test_products_with_a_staged_epilogue(M, N, Kd):
    K = _k()
    x, w = _rand(M, Kd + 8, dtype=BF, seed=1)[:, :Kd], _rand(2 * N, Kd, dtype=BF, seed=2, scale=2 * Kd ** -0.5)
    want = _d(x) @ _d(w).t()
    for bn in (0, 128, 256):
        _close(K.gemm_staged(x, w[:N], alpha=0.5, block_n=bn), 0.5 * want[:, :N], BF)
    for act, f in (("gelu", R.gelu), ("silu", R.silu)):
        _close(K.gemm_staged(x, w, act=act), f(want[:, :N]) * want[:, N:], BF)
    assert K.status_fetch() == 0


@pytest.mark.parametrize("dtype", DT)
def test_token_gate(dtype):
    K = _k()
    g, table = _rand(70, 64, dtype=dtype, seed=1, scale=2.0), _rand(11, 150, dtype=dtype, seed=2)
    tok = torch.randint(0, 11, (70,), generator=torch.Generator().manual_seed(0)).int().cuda()
    o = K.token_gate(g, tok, table, 100, 50)
    _close(o[:, :50], R.gelu(_d(g)[:, :50]) * _d(table)[tok.long().cpu(), 100:], dtype)
    assert not bool(o[:, 50:].any())


# ---------------------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_portions_of_all_sizes_match_the_plain_statement(name, dtype):
    U.SUITE.check_portions(name, "cuda", dtype, 300, [[300], [2], [1], [7, 2, 130, 1, 1, 3, 16], [64, 1], [129, 2, 128, 1]])
    assert _k().status_fetch() == 0


@pytest.mark.parametrize("block_size", [1, 8, 24, 32, 96])
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_block_sizes(name, block_size):
    U.SUITE.check_portions(name, "cuda", BF, 210, [[210], [100, 1]], block_size)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "tiles", "choice"])
def test_requests_side_by_side_and_reused_pages(name, dtype):
    U.SUITE.check_interleaved(name, "cuda", dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "tiles", "odd"])
def test_greedy_generation_through_the_scheduler(name, dtype):
    U.SUITE.check_generate(name, "cuda", dtype, 12, 32)


def test_requests_that_share_a_batch_do_not_see_each_other():
    U.SUITE.check_generate_matches_decode_of_requests("mixed", "cuda", F32)


@pytest.mark.parametrize("dtype", DT)
def test_long_decoding(dtype):
    """Decoding far past every window, over many pages, each token from the pages the earlier ones left."""
    cfg = U.CONFIGS["tiles"]
    w = U.weights(cfg, 9)
    toks = U.tokens(cfg, 700, 4)
    model, sched = U.server(U.engine(cfg, w, "cuda", dtype), blocks=64)
    got = U.run_portions(model, sched, 0, toks, [3, 1])
    e = U.error(got, U.SUITE.reference(cfg, w, toks))
    assert e < U.TOL[dtype], e


def test_a_wide_batch_decodes_like_each_alone():
    """More sequences than one block of rows of any product."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, 11)
    eng = U.engine(cfg, w, "cuda", BF)
    model, sched = U.server(eng, blocks=400, slots=140)
    seqs = [U.tokens(cfg, 3 + n % 40, n) for n in range(140)]
    for n, s in enumerate(seqs):
        sched.feed(model, [(n, s[:-1], [])])
    got = sched.feed(model, [(n, s[-1:], [0]) for n, s in enumerate(seqs)])
    want = torch.stack([U.SUITE.reference(cfg, w, s)[-1] for s in seqs])
    assert U.error(torch.cat(got), want) < U.TOL[BF]


def test_results_do_not_depend_on_pages():
    cfg = U.CONFIGS["tiles"]
    w = U.weights(cfg, 12)
    eng = U.engine(cfg, w, "cuda", BF)
    toks = U.tokens(cfg, 150, 5)
    outs = []
    for bs, others in ((16, 0), (16, 2), (32, 1), (96, 1)):
        model, sched = U.server(eng, blocks=64, slots=4, block_size=bs)
        for o in range(others):
            sched.feed(model, [(50 + o, U.tokens(cfg, 40 + o, o), [])])
        if others == 2:
            sched.end_session(50)
        outs.append(U.run_portions(model, sched, 0, toks, [60, 1, 1, 50, 1]))
    assert all(torch.equal(outs[0], o) for o in outs[1:])
