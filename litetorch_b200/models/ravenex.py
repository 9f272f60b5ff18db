"""Ravenex: a decoder of latent-attention layers.  Every layer has

* windowed attention whose keys and values are linear maps of a small normed latent plus one rotated key part shared by all
  heads; only these two are cached, and a layer may read the ones of an earlier layer (`kv_from`);
* a dense gated feed-forward (GELU), a mixture of experts (sigmoid router with a correction that takes part in the choice
  only, plus a shared expert), or none;
* an input of its own per token: a slice of a second embedding, gated by the residual.

Each of them is normed before and after and joins the fp32 residual with one multiplier.  This module holds the
configuration (read from `config.json`), the tensor names and shapes of a checkpoint, and the engine: the weights in the
form the kernels want them.  The step functions are in `ravenex_serving`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from .llama import kernels_for
from .rotary import RotaryConfig
from .weights import checked_fetch, pad_dim, round_up, stack_rows


@dataclass
class LatentAttentionConfig:
    heads: int
    dim: int                          # unrotated query / key size of a head
    rot_dim: int
    vdim: int
    kv_rank: int
    window: int                       # 0: every earlier key
    scale: float
    rot: RotaryConfig
    kv_from: Optional[int] = None     # the layer whose latents are read; None: this layer's own


@dataclass
class GluConfig:
    ff: int


@dataclass
class MoeConfig:
    experts: int
    top: int
    ff: int
    shared: Optional[GluConfig]


@dataclass
class RavenexLayerConfig:
    mixer: LatentAttentionConfig
    mlp: object                       # GluConfig, MoeConfig or None


@dataclass
class RavenexConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    side_dim: int                     # size of a layer's slice of the second embedding; 0: none
    layers: List[RavenexLayerConfig]
    max_seq: Optional[int] = None     # positions have no end

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def parse(c: dict) -> "RavenexConfig":
        """From the dict of a `config.json`."""
        layers: List[RavenexLayerConfig] = []
        for i, e in enumerate(c["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError("layer %d: unknown type %r" % (i, e["type"]))
            m = e["mixer"]
            a = LatentAttentionConfig(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                      int((m.get("mask") or {}).get("size") or 0), float(m["scale"]), RotaryConfig.parse(m.get("rot")),
                                      None if m.get("kv_from") is None else int(m["kv_from"]))
            if a.rot.dims != a.rot_dim or a.rot_dim % 2:
                raise ValueError("layer %d: the rotation covers %d dimensions, the rotated part has %d" % (i, a.rot.dims, a.rot_dim))
            if a.kv_from is not None:
                src = layers[a.kv_from].mixer if 0 <= a.kv_from < i else None
                if src is None or src.kv_from is not None or (src.kv_rank, src.rot_dim, src.rot) != (a.kv_rank, a.rot_dim, a.rot):
                    raise ValueError("layer %d cannot read the latents of layer %d" % (i, a.kv_from))
            mlp = e.get("mlp")
            if mlp is not None:
                if mlp["kind"] == "dense":
                    mlp = GluConfig(int(mlp["ff"]))
                elif mlp["kind"] == "moe":
                    sh = mlp.get("shared")
                    mlp = MoeConfig(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]),
                                    GluConfig(int(sh["ff"])) if sh else None)
                    if not 1 <= mlp.top <= mlp.experts:
                        raise ValueError("layer %d: %d of %d experts" % (i, mlp.top, mlp.experts))
                else:
                    raise ValueError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))
            layers.append(RavenexLayerConfig(a, mlp))
        side = c.get("token_side")
        return RavenexConfig(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["residual_mult"]),
                             int(side["dim"]) if side else 0, layers)


def tensor_shapes(cfg: RavenexConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint."""
    W = cfg.width
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W)}
    if cfg.side_dim:
        t["side.embed"] = (cfg.vocab, cfg.side_dim * len(cfg.layers))

    def glu(p, ff):
        t.update({p + "gate": (ff, W), p + "up": (ff, W), p + "down": (W, ff)})

    for i, lay in enumerate(cfg.layers):
        p, a, f = "l%d." % i, lay.mixer, lay.mlp
        m = p + "mix."
        t.update({p + "norm1": (W,), p + "norm1b": (W,), m + "q": (a.heads * (a.dim + a.rot_dim), W), m + "uk": (a.heads * a.dim, a.kv_rank),
                  m + "uv": (a.heads * a.vdim, a.kv_rank), m + "o": (W, a.heads * a.vdim)})
        if a.kv_from is None:
            t.update({m + "dkv": (a.kv_rank + a.rot_dim, W), m + "dkv.norm": (a.kv_rank,)})
        if f is not None:
            t.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if isinstance(f, GluConfig):
            glu(p + "mlp.", f.ff)
        elif isinstance(f, MoeConfig):
            t.update({p + "mlp.router": (f.experts, W), p + "mlp.correction": (f.experts,)})
            for e in range(f.experts):
                glu(p + "mlp.e%d." % e, f.ff)
            if f.shared:
                glu(p + "mlp.shared.", f.shared.ff)
        if cfg.side_dim:
            t.update({p + "side.gate": (cfg.side_dim, W), p + "side.proj": (W, cfg.side_dim), p + "side.norm": (W,)})
    t["final.norm"] = (W,)
    t["head"] = (cfg.vocab, W)
    return t


def random_tensor(name: str, shape, gen: torch.Generator, device="cpu", dtype=torch.bfloat16) -> torch.Tensor:
    """Random values of a sensible size for the tensor of this name."""
    leaf = name.rsplit(".", 1)[-1]
    z = torch.randn(shape, generator=gen, device=device)
    if leaf.startswith("norm"):
        z = 1.0 + 0.1 * z
    elif leaf == "correction":
        z = 0.1 * z
    elif leaf != "embed":                             # a matrix [out, in]
        z = z / math.sqrt(shape[-1])
    return z.to(dtype)


class GluWeights:
    """A gated feed-forward: gate and up stacked, the inner size padded with zeros to a multiple of 32."""

    def __init__(self, get, p: str, ff: int):
        n = round_up(ff, 32)
        self.gu = torch.cat([pad_dim(get(p + "gate"), 0, n), pad_dim(get(p + "up"), 0, n)])
        self.down = pad_dim(get(p + "down"), 1, n)


class MoeWeights:
    """The experts' matrices behind one another: gu [experts, 2 n, width] (gate rows, then up rows), down [experts, width, n]."""

    def __init__(self, get, p: str, cfg: MoeConfig, width: int):
        self.cfg = cfg
        self.router, self.correction = get(p + "router"), get(p + "correction", torch.float32)
        n = round_up(cfg.ff, 32)
        opt = dict(dtype=self.router.dtype, device=self.router.device)
        self.gu, self.down = torch.zeros(cfg.experts, 2 * n, width, **opt), torch.zeros(cfg.experts, width, n, **opt)
        for e in range(cfg.experts):
            q = p + "e%d." % e
            self.gu[e, :cfg.ff], self.gu[e, n:n + cfg.ff] = get(q + "gate"), get(q + "up")
            self.down[e, :, :cfg.ff] = get(q + "down")
        self.shared = GluWeights(get, p + "shared.", cfg.shared.ff) if cfg.shared else None


class LatentAttentionWeights:
    """Matrices of a latent-attention layer with every head's parts padded with zeros to the sizes the kernels run on:
    `d` unrotated and `r` rotated query / key columns, `v` value columns, latents of `c` columns.

    w_in   [heads (d + r) | latent, rotated key part, width]   one product for all that reads the layer's input
    w_kv   [heads d | heads v, c]                              keys and values of a latent (prompts)
    w_qk   [heads, c, d]                                       the unrotated query moved to the latent's side (decoding)
    w_v    [heads, v, c]                                       values of a sum of latents (decoding); shares memory with w_kv
    """

    def __init__(self, cfg: LatentAttentionConfig, get, p: str, device, dtype):
        a = cfg
        # what the tensor-core kernels take; on the CPU their twins run the same forms
        latent_tc = (torch.device(device).type == "cpu" or dtype == torch.bfloat16) and a.kv_rank <= 512 and a.rot_dim <= 64
        self.tensor_cores = latent_tc and a.dim <= 128 and a.vdim <= 128
        big, small = (64 if latent_tc else 8), (64 if self.tensor_cores else 8)
        self.c, self.r = round_up(a.kv_rank, big), round_up(a.rot_dim, big)   # as in the cache: equal for all layers that share it
        self.d, self.v = round_up(a.dim, small), round_up(a.vdim, small)
        if self.tensor_cores and self.d == 128:
            self.v = 128                                                      # the kernel for the larger keys has one value size
        H = a.heads
        q = get(p + "q")
        W = q.shape[1]
        q = q.view(H, a.dim + a.rot_dim, W)
        q = torch.cat([pad_dim(q[:, :a.dim], 1, self.d), pad_dim(q[:, a.dim:], 1, self.r)], 1).reshape(H * (self.d + self.r), W)
        if a.kv_from is None:
            self.w_in, (_, self.c_off) = stack_rows([q, get(p + "dkv")])
            self.c_norm = get(p + "dkv.norm", torch.float32)
        else:
            self.w_in, _ = stack_rows([q])
            self.c_off, self.c_norm = -1, None
        uk = pad_dim(pad_dim(get(p + "uk").view(H, a.dim, a.kv_rank), 1, self.d), 2, self.c)
        uv = pad_dim(pad_dim(get(p + "uv").view(H, a.vdim, a.kv_rank), 1, self.v), 2, self.c)
        self.w_kv = torch.cat([uk.reshape(H * self.d, self.c), uv.reshape(H * self.v, self.c)])
        self.w_qk = uk.transpose(1, 2).contiguous()
        self.w_v = self.w_kv[H * self.d:].view(H, self.v, self.c)
        self.o = pad_dim(get(p + "o").view(W, H, a.vdim), 2, self.v).reshape(W, H * self.v)
        freq, self.rot_gain = a.rot.frequencies()
        self.freq = torch.tensor(freq or [0.0], dtype=torch.float64, device=device)


class RavenexLayer:
    """One layer's weights: matrices that share an input fused, everything that enters 32-bit arithmetic as fp32."""

    def __init__(self, cfg: RavenexLayerConfig, side_dim: int, get, p: str, device, dtype):
        f32 = torch.float32
        self.cfg = cfg
        self.norm1, self.norm1b = get(p + "norm1", f32), get(p + "norm1b", f32)
        self.mix = LatentAttentionWeights(cfg.mixer, get, p + "mix.", device, dtype)
        self.mlp = None
        if cfg.mlp is not None:
            self.norm2, self.norm2b = get(p + "norm2", f32), get(p + "norm2b", f32)
            if isinstance(cfg.mlp, MoeConfig):
                self.mlp = MoeWeights(get, p + "mlp.", cfg.mlp, self.norm1.numel())
            else:
                self.mlp = GluWeights(get, p + "mlp.", cfg.mlp.ff)
        if side_dim:
            n = round_up(side_dim, 32)
            self.side_gate, self.side_proj = pad_dim(get(p + "side.gate"), 0, n), pad_dim(get(p + "side.proj"), 1, n)
            self.side_norm = get(p + "side.norm", f32)


class RavenexEngine:
    """Configuration and weights on one device.  dtype: bf16 (matrices and activations; what the model computes in 32-bit
    stays fp32) or fp32 (everything in true fp32)."""

    def __init__(self, cfg: RavenexConfig, tensors, device="cuda", dtype=torch.bfloat16):
        """tensors: a mapping, or a function name -> tensor."""
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        if dtype not in (torch.bfloat16, torch.float32):
            raise TypeError("weights run in bfloat16 or float32, not %s" % dtype)
        self.K = kernels_for(self.device)
        get = checked_fetch(tensors, tensor_shapes(cfg), self.device, dtype)
        self.embed, self.head = get("embed"), get("head")
        self.side_embed = get("side.embed") if cfg.side_dim else None
        self.final_norm = get("final.norm", torch.float32)
        self.layers = [RavenexLayer(lay, cfg.side_dim, get, "l%d." % i, self.device, dtype) for i, lay in enumerate(cfg.layers)]

    @staticmethod
    def from_directory(directory: str, config: dict, device="cuda", dtype=torch.bfloat16) -> "RavenexEngine":
        from .llama_io import read_state_dict
        return RavenexEngine(RavenexConfig.parse(config), read_state_dict(directory), device, dtype)

    @staticmethod
    def random(cfg: RavenexConfig, device="cuda", dtype=torch.bfloat16, seed: int = 0) -> "RavenexEngine":
        shapes = tensor_shapes(cfg)
        gen = torch.Generator(device=device).manual_seed(seed)
        return RavenexEngine(cfg, lambda n: random_tensor(n, shapes[n], gen, device), device, dtype)
