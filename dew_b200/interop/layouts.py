"""Copying a release's tensors into parameters that join several of them (fused projections, stacked experts), for designs whose ``config.json``
describes every layer by itself."""
from __future__ import annotations

from typing import List, Mapping, Sequence, Tuple

import torch

Table = Sequence[Tuple[torch.Tensor, Tuple[str, ...]]]


def copy_tensors(table: Table, tensors: Mapping[str, torch.Tensor], strict: bool = True, spare: Tuple[str, ...] = ()) -> List[str]:
    """``table``: every parameter (or a slice of one, whose first axis may stand split in two) with the release's tensors that make it up, joined along
    their first axis.  Returns the names
    nothing read, those that start with a ``spare`` prefix aside (raises on them with ``strict``)."""
    read = set()
    for p, names in table:
        parts = [tensors[n] for n in names]
        t = parts[0] if len(parts) == 1 else torch.cat(parts, 0)
        if p.dim() == t.dim() + 1 and p.shape[0] * p.shape[1] == t.shape[0] and p.shape[2:] == t.shape[1:]:
            t = t.reshape(p.shape)
        if tuple(t.shape) != tuple(p.shape):
            raise ValueError(f"{' | '.join(names)}: shape {tuple(t.shape)} on disk does not fit the parameter's {tuple(p.shape)}")
        with torch.no_grad():
            p.copy_(t.to(p.dtype))
        read.update(names)
    left = sorted(k for k in tensors if k not in read and not (spare and k.startswith(spare)))
    if strict and left:
        raise KeyError(f"{len(left)} tensor(s) of the release were not read: {left[:6]}")
    return left
