"""Safuvik: a decoder whose residual is carried by several hyper-connected streams and whose layers are of two kinds,

* `parallel`: windowed grouped-query attention (norm over the whole q / k projection, interleaved rotary embedding with
  YaRN scaling, one sigmoid gate per head) beside a recurrent block (short convolution, gated linear recurrence, GELU
  branch); the two outputs are RMS-normed and averaged;
* `mlstm`: a matrix memory with exponential gates;

each followed by a clamped gated feed-forward, or by none.  This module holds the configuration (read from `config.json`),
the tensor names and shapes of a checkpoint, and the engine: the weights in the form the kernels want them.  The step
functions are in `safuvik_serving`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from .llama import kernels_for
from .rotary import RotaryConfig
from .weights import checked_fetch, stack_rows


@dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    rot: RotaryConfig


@dataclass
class RecurrentConfig:
    width: int
    blocks: int
    conv: int


@dataclass
class ParallelConfig:
    left: AttentionConfig
    right: RecurrentConfig


@dataclass
class MlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass
class MlpConfig:
    ff: int
    limit: float


@dataclass
class LayerConfig:
    mixer: object                     # ParallelConfig or MlstmConfig
    mlp: Optional[MlpConfig]


@dataclass
class SafuvikConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    logit_scale: float
    layers: List[LayerConfig]
    max_seq: Optional[int] = None     # positions have no end

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def parse(c: dict) -> "SafuvikConfig":
        """From the dict of a `config.json`."""
        layers = []
        for i, e in enumerate(c["layers"]):
            m = e["mixer"]
            if e["type"] == "parallel":
                a, r = m["left"], m["right"]
                mixer = ParallelConfig(
                    AttentionConfig(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), int(a["mask"]["size"]),
                                    float(a["scale"]), RotaryConfig.parse(a.get("rot"))),
                    RecurrentConfig(int(r["width"]), int(r["blocks"]), int(r["conv"])))
            elif e["type"] == "mlstm":
                mixer = MlstmConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
            else:
                raise ValueError("layer %d: unknown type %r" % (i, e["type"]))
            mlp = e.get("mlp")
            if mlp is not None:
                if mlp["kind"] != "dense":
                    raise ValueError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))
                mlp = MlpConfig(int(mlp["ff"]), float(mlp["limit"]))
            layers.append(LayerConfig(mixer, mlp))
        return SafuvikConfig(int(c["vocab"]), int(c["width"]), int(c["streams"]), float(c["norm"]["eps"]), float(c["logit_scale"]), layers)


def tensor_shapes(cfg: SafuvikConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a checkpoint."""
    W, S = cfg.width, cfg.streams
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W)}
    for i, lay in enumerate(cfg.layers):
        p = "l%d." % i
        t[p + "norm1"] = (W,)
        m, x = p + "mix.", lay.mixer
        if isinstance(x, ParallelConfig):
            a, r = x.left, x.right
            bw = r.width // r.blocks
            l, g = m + "left.", m + "right."
            t.update({l + "q": (a.heads * a.dim, W), l + "k": (a.kv_heads * a.dim, W), l + "v": (a.kv_heads * a.vdim, W),
                      l + "q.norm": (a.heads * a.dim,), l + "k.norm": (a.kv_heads * a.dim,), l + "g": (a.heads, W),
                      l + "o": (W, a.heads * a.vdim), l + "out": (W,),
                      g + "y": (r.width, W), g + "y.b": (r.width,), g + "x": (r.width, W), g + "x.b": (r.width,),
                      g + "conv": (r.width, r.conv), g + "conv.b": (r.width,), g + "ra": (r.blocks, bw, bw), g + "ra.b": (r.blocks, bw),
                      g + "ri": (r.blocks, bw, bw), g + "ri.b": (r.blocks, bw), g + "lam": (r.width,), g + "o": (W, r.width), g + "out": (W,)})
        else:
            hd, he = x.heads * x.dim, x.heads * x.vdim
            t.update({m + "q": (hd, W), m + "k": (hd, W), m + "v": (he, W), m + "g": (he, W), m + "o": (W, he), m + "norm": (he,),
                      m + "i": (x.heads, W), m + "i.b": (x.heads,), m + "f": (x.heads, W), m + "f.b": (x.heads,)})
        if lay.mlp is not None:
            t.update({p + "norm2": (W,), p + "mlp.gate": (lay.mlp.ff, W), p + "mlp.up": (lay.mlp.ff, W), p + "mlp.down": (W, lay.mlp.ff)})
        for q in (1, 2) if lay.mlp is not None else (1,):
            t.update({p + "hc%d.in" % q: (S,), p + "hc%d.out" % q: (S,), p + "hc%d.mix" % q: (S, S)})
    t["final.norm"] = (W,)
    t["head"] = (cfg.vocab, W)
    return t


def random_tensor(name: str, shape, gen: torch.Generator, device="cpu", dtype=torch.bfloat16) -> torch.Tensor:
    """Random values of a sensible size for the tensor of this name."""
    leaf = name.rsplit(".", 1)[-1]
    z = torch.randn(shape, generator=gen, device=device)
    if leaf.startswith("norm") or name.endswith(".norm") or (leaf == "out" and ".mix." in name):
        z = 1.0 + 0.1 * z
    elif ".hc" in name:
        s = shape[0]
        base = {"in": 1.0 / s, "out": 1.0}.get(leaf)
        z = 0.1 / s * z + (base if base is not None else 0.9 * torch.eye(s, device=device))
    elif leaf == "lam":
        z = -3.0 + z
    elif name.endswith("mix.f.b"):
        z = 3.0 + z
    elif leaf == "b":
        z = 0.1 * z
    elif leaf == "embed":
        pass
    else:                                             # a matrix [.., out, in] or a convolution [channels, taps]
        z = z / math.sqrt(shape[-1])
    return z.to(dtype)


class HyperWeights:
    def __init__(self, get, p: str):
        self.inn, self.out, self.mix = get(p + "in", torch.float32), get(p + "out", torch.float32), get(p + "mix", torch.float32)


class SafuvikLayer:
    """One layer's weights: matrices that share an input fused, everything that enters 32-bit arithmetic as fp32."""

    def __init__(self, cfg: LayerConfig, get, p: str, device):
        f32 = torch.float32
        self.cfg = cfg
        self.norm1, self.hc1 = get(p + "norm1", f32), HyperWeights(get, p + "hc1.")
        m, x = p + "mix.", cfg.mixer
        if isinstance(x, ParallelConfig):
            l, r = m + "left.", m + "right."
            self.w_in, self.offs = stack_rows([get(l + "q"), get(l + "k"), get(l + "v"), get(l + "g"), get(r + "y"), get(r + "x")])
            self.q_norm, self.k_norm = get(l + "q.norm", f32), get(l + "k.norm", f32)
            self.left_o, self.left_out = get(l + "o"), get(l + "out", f32)
            freq, self.rot_gain = x.left.rot.frequencies()
            self.freq = torch.tensor(freq or [0.0], dtype=torch.float64, device=device)
            self.y_b, self.x_b = get(r + "y.b", f32), get(r + "x.b", f32)
            self.conv, self.conv_b = get(r + "conv", f32), get(r + "conv.b", f32)
            self.gates = torch.cat([get(r + "ra"), get(r + "ri")], 1).contiguous()          # [blocks, rows of r | rows of i, in]
            self.r_b, self.i_b = get(r + "ra.b", f32), get(r + "ri.b", f32)
            self.decay = torch.nn.functional.softplus(get(r + "lam", torch.float64)).float()
            self.right_o, self.right_out = get(r + "o"), get(r + "out", f32)
        else:
            self.w_in, self.offs = stack_rows([get(m + "q"), get(m + "k"), get(m + "v"), get(m + "g")])
            self.w_if = torch.cat([get(m + "i"), get(m + "f")]).contiguous()
            self.i_b, self.f_b = get(m + "i.b", f32), get(m + "f.b", f32)
            self.head_norm, self.o = get(m + "norm", f32), get(m + "o")
        if cfg.mlp is not None:
            self.norm2, self.hc2 = get(p + "norm2", f32), HyperWeights(get, p + "hc2.")
            self.w_gu = torch.cat([get(p + "mlp.gate"), get(p + "mlp.up")]).contiguous()
            self.w_down = get(p + "mlp.down")


class SafuvikEngine:
    """Configuration and weights on one device.  dtype: bf16 (matrices and activations; what the model computes in 32-bit
    stays fp32) or fp32 (everything in true fp32)."""

    def __init__(self, cfg: SafuvikConfig, tensors, device="cuda", dtype=torch.bfloat16):
        """tensors: a mapping, or a function name -> tensor (called once per name, so that a big random model need never
        exist twice)."""
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        if dtype not in (torch.bfloat16, torch.float32):
            raise TypeError("weights run in bfloat16 or float32, not %s" % dtype)
        self.K = kernels_for(self.device)
        get = checked_fetch(tensors, tensor_shapes(cfg), self.device, dtype)
        self.embed, self.head = get("embed"), get("head")
        self.final_norm = get("final.norm", torch.float32)
        self.layers = [SafuvikLayer(lay, get, "l%d." % i, self.device) for i, lay in enumerate(cfg.layers)]

    @staticmethod
    def from_directory(directory: str, config: dict, device="cuda", dtype=torch.bfloat16) -> "SafuvikEngine":
        from .llama_io import read_state_dict
        return SafuvikEngine(SafuvikConfig.parse(config), read_state_dict(directory), device, dtype)

    @staticmethod
    def random(cfg: SafuvikConfig, device="cuda", dtype=torch.bfloat16, seed: int = 0) -> "SafuvikEngine":
        shapes = tensor_shapes(cfg)
        gen = torch.Generator(device=device).manual_seed(seed)
        return SafuvikEngine(cfg, lambda n: random_tensor(n, shapes[n], gen, device), device, dtype)
