"""Bringing the tensors of a checkpoint into the form the kernels want: shape checks, matrices that share an input stacked
into one product, and padding."""
from __future__ import annotations

from typing import Callable, Dict, List, Tuple

import torch


def checked_fetch(tensors, shapes: Dict[str, Tuple[int, ...]], device, dtype) -> Callable:
    """get(name, as_dtype=None): the tensor of that name on `device`, its shape checked.  tensors: a mapping, or a function
    name -> tensor (called once per name, so that a big random model need never exist twice)."""
    fetch = tensors if callable(tensors) else tensors.__getitem__

    def get(name, as_dtype=None):
        try:
            t = fetch(name)
        except KeyError:
            raise KeyError("the checkpoint has no tensor %r" % name) from None
        if tuple(t.shape) != tuple(shapes[name]):
            raise ValueError("%s: the checkpoint gives %s, the configuration expects %s" % (name, tuple(t.shape), tuple(shapes[name])))
        return t.to(device).to(as_dtype or dtype).contiguous()
    return get


def round_up(n: int, to: int) -> int:
    return (n + to - 1) // to * to


def stack_rows(ws: List[torch.Tensor]) -> Tuple[torch.Tensor, List[int]]:
    """Matrices with the same input stacked by rows, every one starting at a multiple of 8 and the whole a multiple of 64
    rows (zeros between): one product whose columns are aligned for vector loads."""
    offs, parts, at = [], [], 0
    for j, w in enumerate(ws):
        offs.append(at)
        end = at + w.shape[0]
        to = round_up(end, 8 if j + 1 < len(ws) else 64)
        parts.append(torch.nn.functional.pad(w, (0, 0, 0, to - end)))
        at = to
    return torch.cat(parts).contiguous(), offs


def pad_dim(t: torch.Tensor, dim: int, to: int) -> torch.Tensor:
    """Zeros behind dimension `dim` up to size `to`."""
    if t.shape[dim] == to:
        return t
    size = list(t.shape)
    size[dim] = to - t.shape[dim]
    return torch.cat([t, t.new_zeros(size)], dim)
