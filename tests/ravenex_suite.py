"""Small Ravenex models for the CPU and the GPU tests, compared with the plain statement in `ravenex_ref`."""
import torch

import ravenex_ref as R
from decoder_suite import TOL, Suite, error, row_errors, run_portions, server, tokens, write_model          # noqa: F401  (used through this module)
from litetorch_b200.models.ravenex import RavenexConfig, RavenexEngine, random_tensor, tensor_shapes


def layer(heads, dim, rot_dim, vdim, rank, window, mlp, scale=None, base=700.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot_dim) ** -0.5,
         "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def config(vocab, width, layers, side=None, eps=1e-5, mult=1.0):
    return {"architecture": "Ravenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "token_side": {"dim": side} if side else None, "layers": layers}


# Where an expert is one of all that are chosen anyway, no rounding can change the choice: those models compare tightly in bf16 too.
CONFIGS = {
    # unequal sizes everywhere; latents read by a later layer with other heads, sizes and window, and across a layer between them;
    # a layer without feed-forward; windows below, at and above a page; one layer that sees everything
    "mixed": config(131, 96, [
        layer(3, 20, 12, 28, 40, 37, dense(72)),
        layer(2, 24, 32, 40, 56, 16, moe(3, 3, 24, 40)),
        layer(5, 36, 12, 20, 40, 60, None, scale=0.3, kv_from=0),
        layer(2, 16, 8, 48, 24, None, moe(2, 2, 40), base=50.0)], side=20, eps=1e-4, mult=0.7),
    # sizes of the tensor-core kernels: keys of 128 + 64 columns, a second pair of layers on 64 + 64, windows about a tile
    "tiles": config(256, 128, [
        layer(4, 128, 64, 64, 128, 129, dense(192), base=20.0),
        layer(17, 64, 64, 128, 128, 64, moe(4, 4, 64, 128), kv_from=0, base=20.0),
        layer(2, 64, 32, 64, 512, 200, moe(2, 2, 96, 32))], side=32, mult=0.4),
    # nothing is a multiple of 8; a rotated part of one pair; no second embedding
    "odd": config(77, 60, [
        layer(3, 10, 6, 5, 21, 23, dense(35)),
        layer(1, 7, 2, 9, 13, 5, moe(5, 5, 11, 17))], eps=1e-3, mult=1.3),
    # head sizes beyond the tensor-core kernels beside sizes within them, on each other's latents; a latent beyond them
    "wide": config(64, 64, [
        layer(2, 144, 16, 130, 48, 50, dense(48)),
        layer(2, 32, 16, 16, 48, 33, None, kv_from=0),
        layer(1, 16, 96, 16, 40, 21, dense(40), base=300.0),
        layer(1, 24, 8, 24, 520, 40, None)], side=5, mult=0.5),
    # a real choice: few of many experts, top 1 as well
    "choice": config(90, 64, [
        layer(2, 16, 16, 16, 32, 40, moe(12, 2, 32, 24)),
        layer(2, 16, 16, 16, 32, 25, moe(40, 5, 16), kv_from=0),
        layer(2, 16, 16, 16, 32, 70, moe(6, 1, 48, 64))], side=8, mult=0.6),
}


def weights(cfg, seed=0):
    """bf16 tensors.  Queries are scaled so that single scores stand out, which a wrong key, a window that is off by one or a
    wrong rotation cannot hide behind; router logits and corrections are spread so that the correction changes choices."""
    gen = torch.Generator().manual_seed(seed)
    w = {n: random_tensor(n, s, gen) for n, s in tensor_shapes(RavenexConfig.parse(cfg)).items()}
    for n in w:
        f = 2.0 if n.endswith("mix.q") else 2.0 if n.endswith(("router", "correction")) else 0
        if f:
            w[n] = (w[n].float() * f).to(torch.bfloat16)
    return w


def engine(cfg, w, device, dtype):
    return RavenexEngine(RavenexConfig.parse(cfg), w, device, dtype)


def measure(got, want, cfg, dtype):
    """bf16 rounding may turn a close choice of experts, which moves that token's logits by a whole expert: where there is a
    choice, the error in bf16 is the median of the rows."""
    if dtype == torch.float32 or not any(m["kind"] == "moe" and m["router"]["top"] < m["router"]["experts"] for m in (x["mlp"] for x in cfg["layers"]) if m):
        return error(got, want)
    return float(row_errors(got, want).median())


SUITE = Suite(CONFIGS, weights, engine, R.forward, measure)
