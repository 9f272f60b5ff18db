"""Small Safuvik models for the CPU and the GPU tests, compared with the plain statement in `safuvik_ref`."""
import torch

import safuvik_ref as R
from decoder_suite import ServingScheduler, Suite, error, run_portions, server, tokens, write_model          # noqa: F401  (used through this module)
from litetorch_b200.models.safuvik import SafuvikConfig, SafuvikEngine, random_tensor, tensor_shapes


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


SUITE = Suite(CONFIGS, weights, engine, R.forward)
reference, check_portions, check_interleaved, check_generate = SUITE.reference, SUITE.check_portions, SUITE.check_interleaved, SUITE.check_generate


def check_generate_matches_decode_of_requests(device, dtype):
    SUITE.check_generate_matches_decode_of_requests("mixed", device, dtype)
