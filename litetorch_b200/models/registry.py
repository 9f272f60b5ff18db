"""Model families and what serving needs of each: how to tell one by its `config.json`, how to load a directory, and how to
put an engine behind a cache.  `load_engine` and `new_serving` are what the server, the examples and `generate` call; a new
family is one more `register`.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict

import torch


@dataclass
class ModelFamily:
    name: str
    matches: Callable[[dict], bool]                 # on the dict of config.json
    load: Callable                                  # (directory, config dict, device, dtype) -> engine
    is_engine: Callable[[object], bool]
    serving: Callable                               # (engine, num_blocks, block_size, max_num_seqs, ...) -> ServingModel
    dtypes: tuple = (torch.bfloat16,)               # what its kernels run on a GPU
    components: tuple = ("all",)                    # native source sets its kernels come from (`_native.COMPONENTS`)


FAMILIES: Dict[str, ModelFamily] = {}


def register(family: ModelFamily) -> ModelFamily:
    FAMILIES[family.name] = family
    return family


def read_config(directory: str) -> dict:
    with open(os.path.join(directory, "config.json")) as f:
        return json.load(f)


def family_of(config: dict) -> ModelFamily:
    for f in FAMILIES.values():
        if f.matches(config):
            return f
    raise ValueError("no model family for this configuration (architecture %r); known: %s" %
                     (config.get("architecture") or config.get("architectures") or config.get("model_type"), ", ".join(sorted(FAMILIES))))


def load_engine(directory: str, device="cuda", dtype=torch.bfloat16):
    """Configuration and weights of a model directory (`config.json` + `*.safetensors`) as an engine.  On the CPU every
    family runs in fp32 whatever `dtype` says."""
    config = read_config(directory)
    fam = family_of(config)
    device = torch.device(device)
    if device.type == "cpu":
        dtype = torch.float32
    elif dtype not in fam.dtypes:
        raise TypeError("%s does not run in %s" % (fam.name, dtype))
    return fam.load(directory, config, device, dtype)


def new_serving(engine, num_blocks: int, block_size: int = 16, max_num_seqs: int = 64, kv_dtype=None, graphs: bool = True,
                prefix_cache_bytes: int = 0):
    """The serving model over an engine: a paged cache of `num_blocks` blocks and, where the family has recurrent layers, a
    state slot for each of `max_num_seqs` sequences."""
    for f in FAMILIES.values():
        if f.is_engine(engine):
            return f.serving(engine, num_blocks=num_blocks, block_size=block_size, max_num_seqs=max_num_seqs, kv_dtype=kv_dtype,
                             graphs=graphs, prefix_cache_bytes=prefix_cache_bytes)
    raise TypeError("no model family serves %r" % type(engine).__name__)


# ---------------------------------------------------------------------------------------------------- Llama
def _is_llama_config(c: dict) -> bool:
    return c.get("model_type") == "llama" or "LlamaForCausalLM" in (c.get("architectures") or [])


def _load_llama(directory, config, device, dtype):
    from . import llama_io
    kw = {}
    if device.type == "cpu":
        from .llama import LocalWeights
        kw["weights"] = LocalWeights(llama_io.config_from_hf(config), "cpu", seed=0, param_dtype=torch.float32)
    return llama_io.load_pretrained(directory, device=device, **kw)


def _is_llama_engine(e) -> bool:
    from .llama import LlamaEngine
    return isinstance(e, LlamaEngine)


def _serve_llama(engine, num_blocks, block_size, max_num_seqs, kv_dtype, graphs, prefix_cache_bytes):
    from .llama_serving import LlamaKVModel
    if kv_dtype is None:
        kv_dtype = torch.bfloat16 if engine.device.type == "cuda" else torch.float32
    return LlamaKVModel(engine, num_blocks=num_blocks, block_size=block_size, kv_dtype=kv_dtype, graphs=graphs,
                        prefix_cache_bytes=prefix_cache_bytes)


register(ModelFamily("llama", _is_llama_config, _load_llama, _is_llama_engine, _serve_llama))


# ---------------------------------------------------------------------------------------------------- Safuvik
def _load_safuvik(directory, config, device, dtype):
    from .safuvik import SafuvikEngine
    return SafuvikEngine.from_directory(directory, config, device, dtype)


def _is_safuvik_engine(e) -> bool:
    from .safuvik import SafuvikEngine
    return isinstance(e, SafuvikEngine)


def _serve_safuvik(engine, num_blocks, block_size, max_num_seqs, kv_dtype, graphs, prefix_cache_bytes):
    from .safuvik_serving import SafuvikModel
    if prefix_cache_bytes:
        raise ValueError("prefix reuse keeps cache blocks only; this family's recurrent state is not part of them")
    if kv_dtype is not None and kv_dtype != engine.dtype:
        raise TypeError("this family keeps its keys and values in the activations' type (%s)" % engine.dtype)
    return SafuvikModel(engine, num_blocks=num_blocks, block_size=block_size, max_num_seqs=max_num_seqs, graphs=graphs)


register(ModelFamily("safuvik", lambda c: c.get("architecture") == "Safuvik", _load_safuvik, _is_safuvik_engine, _serve_safuvik,
                     dtypes=(torch.bfloat16, torch.float32), components=("serving", "paged", "simt", "hybrid")))


# ---------------------------------------------------------------------------------------------------- Ravenex
def _load_ravenex(directory, config, device, dtype):
    from .ravenex import RavenexEngine
    return RavenexEngine.from_directory(directory, config, device, dtype)


def _is_ravenex_engine(e) -> bool:
    from .ravenex import RavenexEngine
    return isinstance(e, RavenexEngine)


def _serve_ravenex(engine, num_blocks, block_size, max_num_seqs, kv_dtype, graphs, prefix_cache_bytes):
    from .ravenex_serving import RavenexModel
    if prefix_cache_bytes:
        raise ValueError("prefix reuse keeps keys and values per head; this family caches latents")
    if kv_dtype is not None and kv_dtype != engine.dtype:
        raise TypeError("this family keeps its latents in the activations' type (%s)" % engine.dtype)
    return RavenexModel(engine, num_blocks=num_blocks, block_size=block_size, graphs=graphs)


register(ModelFamily("ravenex", lambda c: c.get("architecture") == "Ravenex", _load_ravenex, _is_ravenex_engine, _serve_ravenex,
                     dtypes=(torch.bfloat16, torch.float32), components=("serving", "simt", "latent")))
