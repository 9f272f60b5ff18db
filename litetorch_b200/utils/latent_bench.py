"""Prompt and decode throughput of Ravenex models beside Llama models of equal size, and their kernels beside each other.

    python bench.py --serving-compare ravenex    (or python -m litetorch_b200.utils.latent_bench [--sizes 1b,8b-layers])

Prompts of `--prompt` tokens, decode steps at position `--context`; how they are timed is in `serving_bench`.  JSON lines, then
tables.
"""
from __future__ import annotations

import torch

from .serving_bench import KernelTable, llama_throughput, run, throughput


def ravenex_config(size: str) -> dict:
    """Layer shapes of current latent-attention models of about the named size (heads of 128 + 64, latents of 512); every other layer
    reads the latents of the one before, all but the first have experts."""
    W, heads, window, layers, ff, experts, top, eff, shared, side = {
        "1b": (2048, 16, 1024, 12, 5632, 16, 4, 512, 1024, 256), "8b-layers": (4096, 32, 2048, 6, 14336, 32, 6, 768, 1536, 256)}[size]
    out = []
    for i in range(layers):
        m = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "mask": {"size": window}, "scale": 192 ** -0.5,
             "rot": {"base": 5e5, "dims": 64}}
        if i % 2:
            m["kv_from"] = i - 1
        mlp = {"kind": "dense", "ff": ff} if i == 0 else {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": eff},
                                                          "shared": {"ff": shared}}
        out.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return {"architecture": "Ravenex", "vocab": 32000, "width": W, "norm": {"eps": 1e-6}, "residual_mult": 0.6, "token_side": {"dim": side},
            "layers": out}


def compare_models(size, prompt, context, batches):
    from ..models import registry
    from ..models.ravenex import RavenexConfig, RavenexEngine, tensor_shapes
    rows = []
    cfg = RavenexConfig.parse(ravenex_config(size))
    params = sum(torch.Size(s).numel() for s in tensor_shapes(cfg).values())
    eng = RavenexEngine.random(cfg, "cuda", torch.bfloat16)
    throughput(lambda nb, B: registry.new_serving(eng, num_blocks=nb, max_num_seqs=B), "ravenex-" + size, params, cfg.vocab, prompt, context, batches, rows)
    del eng
    torch.cuda.empty_cache()
    llama_throughput(size, params, prompt, context, batches, rows)
    return rows


# ---------------------------------------------------------------------------------------------------- kernels
def compare_kernels(size, T, context, B):
    """One row per kernel: (group, design, name, ms, floor ms).  A group holds like kernels of the two designs."""
    from ..models.ravenex import RavenexConfig
    from ..ops import kernels as K
    from .serving_bench import llama_config
    cfg = RavenexConfig.parse(ravenex_config(size))
    lc = llama_config(size, 10 ** 9)
    a, moe, ff = cfg.layers[0].mixer, cfg.layers[1].mlp, cfg.layers[0].mlp.ff
    W, H, d, r, v, c, window, side = cfg.width, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.window, cfg.side_dim
    E, top, eff = moe.experts, moe.top, moe.ff
    Hl, Gl, Dl = lc.n_heads, lc.n_kv_heads, lc.head_dim
    bf = lambda *s: torch.randn(*s, device="cuda", dtype=torch.bfloat16)
    f32 = lambda *s: torch.randn(*s, device="cuda")
    table = KernelTable(size)
    add = table.add
    w1, bs = f32(W), 16
    dt = dict(dtype=torch.bfloat16, mult=0.6)
    freq = torch.tensor(a.rot.frequencies()[0], dtype=torch.float64, device="cuda")
    router, corr = bf(E, W) * W ** -0.5, torch.zeros(E, device="cuda")
    e_gu, e_down = bf(E, 2 * eff, W), bf(E, W, eff)
    for tag, n in (("prompt %d" % T, T), ("decode %d" % B, B)):
        prompt = n == T
        x, h, y = f32(n, W), bf(n, W), bf(n, W)
        add(tag + " norm", "llama", "rmsnorm", lambda: K.norm_fwd(h, w1.bfloat16()), 4.0 * n * W)
        add(tag + " norm", "ravenex", "residual, norm, norm", lambda: K.residual_norm(x, 1e-6, norm=w1, y=y, y_norm=w1, **dt), 12.0 * n * W)
        # products
        for design, name, N, Kd in (("llama", "qkv", (Hl + 2 * Gl) * Dl, W), ("ravenex", "mixer input", H * (d + r) + c + r, W), ("llama", "down", W, ff),
                                    ("ravenex", "attention output", W, H * v), ("ravenex", "shared down", W, moe.shared.ff), ("ravenex", "side gate", side, W),
                                    ("ravenex", "side projection", W, side)):
            xx, ww = bf(n, Kd), bf(N, Kd)
            add(tag + " product", design, name, lambda: K.linear(xx, ww), 2.0 * (n * Kd + N * Kd + n * N), 2.0 * n * N * Kd)
        # rotary and cache write
        nb = ((T if prompt else B * (context + 16)) + bs - 1) // bs + 1
        kc, vc = bf(nb, Gl, bs, Dl), bf(nb, Gl, bs, Dl)
        proj = bf(n, (Hl + 2 * Gl) * Dl)
        pos = (torch.arange(n, device="cuda") if prompt else torch.full((n,), context, device="cuda")).int()
        slots = torch.randperm(nb * bs, device="cuda")[:n].int() if not prompt else torch.arange(n, device="cuda").int()
        cos = torch.randn(1 << 15, Dl // 2, device="cuda")

        def llama_qkv():
            K.rope_(proj, cos, cos, 1, Hl, Dl, col_offset=0, positions=pos)
            K.rope_(proj, cos, cos, 1, Gl, Dl, col_offset=Hl * Dl, positions=pos)
            K.kv_append(proj[:, Hl * Dl:(Hl + Gl) * Dl].reshape(n, Gl, Dl), proj[:, (Hl + Gl) * Dl:].reshape(n, Gl, Dl), kc, vc, slots, bs, False)
        add(tag + " qkv", "llama", "rope x 2, copies, cache write", llama_qkv, 4.0 * n * (Hl + 2 * Gl) * Dl)
        lat = bf(nb, 1, bs, c + r)
        mine = bf(n, H * (d + r) + c + r)
        lin, q_out = bf(n, c + r), bf(n, H, c + r)
        add(tag + " qkv", "ravenex", "rope, latent norm, cache write" + (", linear copy" if prompt else ""),
            lambda: K.latent_rope(mine, H, d, r, r, pos, slots, freq=freq, c_off=H * (d + r), rank=c, c_norm=w1[:c], cache=lat, q_out=None if prompt else q_out,
                                  lin=lin if prompt else None), 4.0 * n * H * r + n * (c + r) * (6.0 if prompt else 4.0))
        if prompt:
            ql, kl, vl = bf(1, n, Hl, Dl), bf(1, n, Gl, Dl), bf(1, n, Gl, Dl)
            add(tag + " attention", "llama", "causal", lambda: K.flash_fwd(ql, kl, vl, causal=True), 4.0 * n * (Hl + Gl) * Dl, 2.0 * Hl * Dl * n * (n + 1))
            wkv = bf(H * (d + v), c)
            add(tag + " product", "ravenex", "keys and values of the latents", lambda: K.linear(lin[:, :c], wkv),
                2.0 * (n * c + wkv.numel() + n * H * (d + v)), 2.0 * n * c * H * (d + v))
            kv = bf(n, H * (d + v))
            q, k, vv = mine[:, :H * (d + r)].unflatten(1, (H, d + r)), kv[:, :H * d].unflatten(1, (H, d)), kv[:, H * d:].unflatten(1, (H, v))
            seen = window * (n - window) + window * (window + 1) / 2 if n > window else n * (n + 1) / 2
            add(tag + " attention", "ravenex", "window %d, shared key part" % window, lambda: K.shared_rope_fwd(q, k, lin[:, c:], vv, scale=0.07, window=window),
                2.0 * n * (H * (d + r) + H * (d + 2 * v) + r), 2.0 * H * (d + r + v) * seen)
        else:
            tables = torch.arange(B * (context // bs + 1), device="cuda").int().view(B, -1).contiguous()
            ctx = torch.full((B,), context, device="cuda").int()
            ql = bf(n, Hl, Dl)
            sp = max(1, min(32, context // 256, (148 * 4 + B * Gl - 1) // (B * Gl)))
            add(tag + " attention", "llama", "paged, context %d" % context, lambda: K.paged_decode(ql, kc, vc, tables, ctx, bs, sp, Dl ** -0.5),
                4.0 * B * context * Gl * Dl)
            seen = min(window, context)
            add(tag + " attention", "ravenex", "latents, window %d" % window,
                lambda: K.latent_decode(q_out, lat, tables, ctx, rank=c, window=window, scale=0.07, max_keys=seen), 2.0 * B * seen * (c + r),
                2.0 * B * seen * H * (2 * c + r))
            wqk, wv = bf(H, c, d), bf(H, v, c)
            qn, ol = mine[:, :H * (d + r)].unflatten(1, (H, d + r))[..., :d], bf(n, H, c)
            add(tag + " product", "ravenex", "query to the latents", lambda: K.head_linear(qn, wqk, out=q_out[..., :c]), 2.0 * (H * c * d + n * H * (c + d)))
            add(tag + " product", "ravenex", "values of the latents", lambda: K.head_linear(ol, wv), 2.0 * (H * v * c + n * H * (c + v)))
        # feed-forward
        gu = bf(n, 2 * ff)
        add(tag + " glu", "llama", "swiglu", lambda: K.swiglu_fwd(gu), 6.0 * n * ff)
        wgu, wd = bf(2 * ff, W), bf(W, ff)
        if prompt:
            add(tag + " glu", "ravenex", "gelu glu", lambda: K.act_glu(gu, "gelu"), 6.0 * n * ff)
        add(tag + " feed-forward", "llama", "gate and up, swiglu, down", lambda: K.gemm(K.swiglu_fwd(K.gemm(h, wgu)), wd), 2.0 * (3 * W * ff + 2 * n * W),
            6.0 * n * W * ff)
        add(tag + " feed-forward", "ravenex", "dense", lambda: K.glu_mlp(h, wgu, wd, "gelu"), 2.0 * (3 * W * ff + 2 * n * W), 6.0 * n * W * ff)
        live = min(E, n * top)
        add(tag + " feed-forward", "ravenex", "%d of %d experts, with router" % (top, E), lambda: K.moe_experts(h, router, corr, top, e_gu, e_down, "silu"),
            2.0 * (3 * W * eff * live + n * W * (1 + top)), 6.0 * n * top * W * eff)
        add(tag + " elementwise", "ravenex", "router logits", lambda: K.moe_logits(h, router), 2.0 * n * W + 4.0 * n * E)
        logits = K.moe_logits(h, router)
        if prompt:
            plan = K.moe_plan(logits, corr, top, 128, h)
            rows = n * top
            add(tag + " elementwise", "ravenex", "choice, slots, rows to slots", lambda: K.moe_plan(logits, corr, top, 128, h), 2.0 * n * W * (1 + top))
            act = K.moe_grouped(plan["xs"], e_gu, plan, "silu")
            add(tag + " product", "ravenex", "experts' gate and up, glu", lambda: K.moe_grouped(plan["xs"], e_gu, plan, "silu"),
                2.0 * (rows * W + e_gu.numel() + 7 * rows * eff), 4.0 * rows * W * eff)
            add(tag + " product", "ravenex", "experts' down", lambda: K.moe_grouped(act, e_down, plan), 2.0 * (rows * eff + e_down.numel() + rows * W),
                2.0 * rows * W * eff)
        else:
            add(tag + " elementwise", "ravenex", "choice and slots", lambda: K.moe_plan(logits, corr, top, 16), 4.0 * n * E)
            plan = dict(K.moe_plan(logits, corr, top, 16), mma=True)
            act = K.moe_grouped(h, e_gu, plan, "silu", picked=True)
            add(tag + " product", "ravenex", "experts' gate and up, glu", lambda: K.moe_grouped(h, e_gu, plan, "silu", picked=True), 2.0 * e_gu.numel() * live / E)
            add(tag + " product", "ravenex", "experts' down", lambda: K.moe_grouped(act, e_down, plan), 2.0 * e_down.numel() * live / E)
        z, slot, weight = K.moe_experts(h, router, corr, top, e_gu, e_down, "silu")
        add(tag + " norm", "ravenex", "experts' rows, residual, norms",
            lambda: K.residual_norm(x, 1e-6, norm=w1, y=y, y_norm=w1, experts=(z, slot, weight), **dt), n * W * (12.0 + 2 * top))
        g, tok, emb = bf(n, side), torch.randint(0, cfg.vocab, (n,), device="cuda").int(), bf(cfg.vocab, side * len(cfg.layers))
        add(tag + " elementwise", "ravenex", "token gate", lambda: K.token_gate(g, tok, emb, side, side), 6.0 * n * side)
    return table.rows


def main(argv=None):
    run(argv, compare_models, compare_kernels)


if __name__ == "__main__":
    main()
