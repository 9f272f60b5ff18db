"""Prompt and decode throughput of Safuvik models beside Llama models of equal size, and their kernels beside each other.

    python bench.py --serving-compare            (or python -m litetorch_b200.utils.hybrid_bench [--sizes 1b,8b-layers])

Prompts of `--prompt` tokens, decode steps at position `--context`; how they are timed is in `serving_bench`.  JSON lines, then
tables.
"""
from __future__ import annotations

import torch

from .serving_bench import KernelTable, llama_throughput, run, throughput


def safuvik_config(size: str) -> dict:
    """Layer shapes of current models of about the named size; three parallel layers to one matrix-memory layer."""
    W, heads, kv, dim, ff, window, layers, mh = {"1b": (2048, 32, 4, 64, 5632, 1024, 16, 4), "8b-layers": (4096, 32, 8, 128, 14336, 2048, 8, 8)}[size]
    mlp = {"kind": "dense", "ff": ff, "limit": 7.0}
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "mask": {"size": window}, "scale": dim ** -0.5,
            "rot": {"base": 5e5, "dims": dim, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    par = {"type": "parallel", "mixer": {"left": left, "right": {"width": W, "blocks": W // 256, "conv": 4}}, "mlp": mlp}
    mat = {"type": "mlstm", "mixer": {"heads": mh, "dim": 256, "vdim": W // mh, "gate_cap": 15.0}, "mlp": mlp}
    return {"architecture": "Safuvik", "vocab": 32000, "width": W, "streams": 4, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [mat if i % 4 == 3 else par for i in range(layers)]}


def compare_models(size, prompt, context, batches):
    from ..models import registry
    from ..models.safuvik import SafuvikConfig, SafuvikEngine, tensor_shapes
    rows = []
    cfg = SafuvikConfig.parse(safuvik_config(size))
    params = sum(torch.Size(s).numel() for s in tensor_shapes(cfg).values())
    eng = SafuvikEngine.random(cfg, "cuda", torch.bfloat16)
    throughput(lambda nb, B: registry.new_serving(eng, num_blocks=nb, max_num_seqs=B), "safuvik-" + size, params, cfg.vocab, prompt, context, batches, rows)
    del eng
    torch.cuda.empty_cache()
    llama_throughput(size, params, prompt, context, batches, rows)
    return rows


# ---------------------------------------------------------------------------------------------------- kernels
def compare_kernels(size, T, context, B):
    """One row per kernel: (group, design, name, ms, floor ms).  A group holds like kernels of the two designs."""
    from ..models.safuvik import SafuvikConfig
    from ..ops import kernels as K
    cfg = SafuvikConfig.parse(safuvik_config(size))
    par, mat = cfg.layers[0].mixer, cfg.layers[3].mixer
    a, r = par.left, par.right
    W, ff, H, G, D, S = cfg.width, cfg.layers[0].mlp.ff, a.heads, a.kv_heads, a.dim, cfg.streams
    C, bw = r.width, r.width // r.blocks
    bf = lambda *s: torch.randn(*s, device="cuda", dtype=torch.bfloat16)
    f32 = lambda *s: torch.randn(*s, device="cuda")
    table = KernelTable(size)
    add = table.add
    w1 = f32(W)
    bs = 16
    for tag, n in (("prompt %d" % T, T), ("decode %d" % B, B)):
        prompt = n == T
        x, h = f32(n, S, W), bf(n, W)
        y, y2 = bf(n, W), bf(n, W)
        wb = bf(W)
        add(tag + " norm", "llama", "rmsnorm", lambda: K.norm_fwd(h, wb), 4.0 * n * W)
        s_in, mix = torch.full((S,), 1.0 / S, device="cuda"), torch.eye(S, device="cuda")
        add(tag + " norm", "safuvik", "streams + norm", lambda: K.hyper_norm(x, w1, 1e-6, dtype=torch.bfloat16, inn=s_in, y=y, mix=mix, out=s_in),
            n * W * (8.0 * S + 4))
        add(tag + " norm", "safuvik", "streams + branch norms + norm",
            lambda: K.hyper_norm(x, w1, 1e-6, dtype=torch.bfloat16, inn=s_in, y=y, y_norm=w1, y2=y2, y2_norm=w1, mix=mix, out=s_in), n * W * (8.0 * S + 6))
        gu = bf(n, 2 * ff)
        add(tag + " glu", "llama", "swiglu", lambda: K.swiglu_fwd(gu), 6.0 * n * ff)
        add(tag + " glu", "safuvik", "clamped glu", lambda: K.clamped_glu(gu, 7.0), 6.0 * n * ff)
        # projections
        for design, name, N, Kd in (("llama", "qkv", (H + 2 * G) * D, W), ("safuvik", "mixer input", (H + 2 * G) * D + 64 + 2 * C, W), ("llama", "down", W, ff),
                                    ("safuvik", "down", W, ff)):
            xx, ww = bf(n, Kd), bf(N, Kd)
            add(tag + " product", design, name, lambda: K.gemm(xx, ww), 2.0 * (n * Kd + N * Kd + n * N), 2.0 * n * N * Kd)
        # rotary and cache write
        nb = ((T if prompt else B * (context + 16)) + bs - 1) // bs + 1
        kc, vc = bf(nb, G, bs, D), bf(nb, G, bs, D)
        proj = bf(n, (H + 2 * G) * D)
        pos = (torch.arange(n, device="cuda") if prompt else torch.full((n,), context, device="cuda")).int()
        slots = torch.randperm(nb * bs, device="cuda")[:n].int() if not prompt else torch.arange(n, device="cuda").int()
        freq, gain = a.rot.frequencies()
        fr = torch.tensor(freq, dtype=torch.float64, device="cuda")
        qn, kn = f32(H * D), f32(G * D)
        cos = torch.randn(1 << 15, D // 2, device="cuda")

        def llama_qkv():
            K.rope_(proj, cos, cos, 1, H, D, col_offset=0, positions=pos)
            K.rope_(proj, cos, cos, 1, G, D, col_offset=H * D, positions=pos)
            K.kv_append(proj[:, H * D:(H + G) * D].reshape(n, G, D), proj[:, (H + G) * D:].reshape(n, G, D), kc, vc, slots, bs, False)
        moved = 4.0 * n * (H + 2 * G) * D
        add(tag + " qkv", "llama", "rope x 2, copies, cache write", llama_qkv, moved)
        lin = bf(2, n, G, D)
        add(tag + " qkv", "safuvik", "norms + rope + cache write" + (" + linear copy" if prompt else ""),
            lambda: K.qkv_rope(proj, 0, H * D, (H + G) * D, H, G, D, D, pos, slots, kc, vc, freq=fr, rot_dims=a.rot.dims, gain=gain, q_norm=qn, k_norm=kn,
                               lin=(lin[0], lin[1]) if prompt else None), moved + (4.0 * n * G * D if prompt else 0))
        q = bf(n, H, D)
        gate = bf(n, H)
        if prompt:
            k, v = bf(1, n, G, D), bf(1, n, G, D)
            w = a.window
            seen = w * (n - w) + w * (w + 1) / 2 if n > w else n * (n + 1) / 2
            add(tag + " attention", "llama", "causal", lambda: K.flash_fwd(q[None], k, v, causal=True), 4.0 * n * (H + G) * D, 4.0 * H * D * n * (n + 1) / 2)
            add(tag + " attention", "safuvik", "window %d" % w, lambda: K.flash_fwd(q[None], k, v, causal=True, window=w), 4.0 * n * (H + G) * D,
                4.0 * H * D * seen)
            add(tag + " elementwise", "safuvik", "head gates", lambda: K.head_gate(q, gate, D), 4.0 * n * H * D)
            # recurrence
            px = bf(n, 2 * C)
            cw, cb, ring, st = f32(C, r.conv), f32(C), f32(r.conv, C), f32(C)
            add(tag + " recurrence", "safuvik", "convolution", lambda: K.conv_causal(px[:, :C], cb, cw, cb, ring, 0), 4.0 * n * C)
            u, gw = bf(n, C), bf(r.blocks, 2 * bw, bw)
            add(tag + " product", "safuvik", "recurrence gates (block diagonal)", lambda: K.block_diag(u, gw), 10.0 * n * C, 4.0 * n * C * bw)
            gl, b2, sp = f32(n, 2 * C), f32(r.blocks, bw), torch.rand(C, device="cuda")
            add(tag + " recurrence", "safuvik", "scan", lambda: K.rglru_scan(u, gl, b2, b2, sp, px[:, C:], cb, px[:, :C], cb, st, ring, r.conv, 0), 14.0 * n * C)
        else:
            tables = torch.arange(B * (context // bs + 1), device="cuda").int().view(B, -1).contiguous()
            ctx = torch.full((B,), context, device="cuda").int()
            sp1 = max(1, min(32, context // 256, (148 * 4 + B * G - 1) // (B * G)))
            add(tag + " attention", "llama", "paged, context %d" % context, lambda: K.paged_decode(q, kc, vc, tables, ctx, bs, sp1, D ** -0.5),
                4.0 * B * context * G * D)
            sp2 = max(1, min(32, a.window // 256, (148 * 4 + B * G - 1) // (B * G)))
            add(tag + " attention", "safuvik", "paged, window %d, gates" % a.window,
                lambda: K.paged_decode(q, kc, vc, tables, ctx, bs, sp2, D ** -0.5, window=a.window, gate=gate, vdim=D), 4.0 * B * min(a.window, context) * G * D)
            px = bf(n, 2 * C)
            cw, cb, ring, st = f32(C, r.conv), f32(C), f32(B, r.conv, C), f32(B, C)
            gw, b2, sp = bf(r.blocks, 2 * bw, bw), f32(r.blocks, bw), torch.rand(C, device="cuda")
            sl = torch.arange(B, device="cuda").int()
            add(tag + " recurrence", "safuvik", "step", lambda: K.rglru_step(px[:, :C], cb, cw, cb, gw, b2, b2, sp, px[:, C:], cb, st, ring, sl, pos),
                4.0 * C * bw + n * C * (6.0 + 8.0 + 4.0 * r.conv), 4.0 * n * C * bw)
        # matrix memory
        mh, md, me = mat.heads, mat.dim, mat.vdim
        p = bf(n, 2 * mh * md + 2 * mh * me)
        cut = (p[:, :mh * md], p[:, mh * md:2 * mh * md], p[:, 2 * mh * md:2 * mh * md + mh * me], p[:, 2 * mh * md + mh * me:])
        lg, gb, hn = f32(n, 2 * mh), torch.full((mh,), 3.0, device="cuda"), f32(mh * me)
        wif = bf(2 * mh, W)
        add(tag + " elementwise", "safuvik", "matrix-memory gate logits", lambda: K.rows_dot(h, wif), 2.0 * n * W)
        if prompt:
            Sm, nm, mm = f32(mh, md, me), f32(2, mh, md), f32(2, mh)
            # per token and head: half a chunk of scores and values, the state applied and updated once
            fl = n * mh * (64 * 2.0 * (md + me) + 4.0 * md * me)
            add(tag + " recurrence", "safuvik", "matrix memory", lambda: K.mlstm_prefill(cut[0], cut[1], cut[2], lg, gb, gb, 15.0, hn, 1e-6, cut[3], Sm, nm, mm, md, me, 0),
                2.0 * n * mh * (2 * md + 3 * me), fl)
        else:
            Sm, nm, mm = f32(B, mh, md, me), f32(B, 2, mh, md), f32(B, 2, mh)
            sl = torch.arange(B, device="cuda").int()
            add(tag + " recurrence", "safuvik", "matrix memory step", lambda: K.mlstm_step(cut[0], cut[1], cut[2], lg, gb, gb, 15.0, hn, 1e-6, cut[3], Sm, nm, mm, sl, pos, md, me),
                8.0 * B * mh * md * me)
    return table.rows


def main(argv=None):
    run(argv, compare_models, compare_kernels)


if __name__ == "__main__":
    main()
