"""Rotary positions of layers that carry their own rotation: which dimensions turn, how they are paired, and by which frequencies.

A call's angles are formed once per rotation (``angles``: cosines and sines of every token, fp32) and shared by every layer and head that turns
the same way; no table over positions exists, so a row may be as long as its cache.  The kernels that apply them sit where the heads pass anyway
(``csrc/kernels/paged_attention.cu``, ``csrc/kernels/latent_attention.cu``); ``turn`` is the plain form.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch

from . import library as L

c_ll, c_int = ctypes.c_longlong, ctypes.c_int


@dataclass(frozen=True)
class Rotary:
    """The first ``dims`` dimensions of a head turn, the rest pass: pair i by ``position * base ** (-2 i / dims) / factor``.  Pairs are the two halves
    of the turned part (i, i + dims / 2), or neighbours (2 i, 2 i + 1) with ``interleaved``."""
    dims: int
    base: float = 10000.0
    interleaved: bool = False
    factor: float = 1.0

    def __post_init__(self):
        if self.dims < 2 or self.dims % 2 or not self.base > 0 or not self.factor > 0:
            raise ValueError(f"a rotation turns an even number of dimensions by positive frequencies, not {self}")

    def frequencies(self) -> torch.Tensor:
        """``[dims / 2]`` in double precision."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        return float(self.base) ** (-2.0 * i / self.dims) / self.factor


_FREQUENCIES: Dict[Tuple[Rotary, torch.device], torch.Tensor] = {}


def _frequencies(rot: Rotary, device: torch.device) -> torch.Tensor:
    key = (rot, device)
    if key not in _FREQUENCIES:
        _FREQUENCIES[key] = rot.frequencies().to(device)
    return _FREQUENCIES[key]


def angles_reference(positions: torch.Tensor, rot: Rotary) -> torch.Tensor:
    a = positions.clamp_min(0).double()[..., None] * _frequencies(rot, positions.device)
    return torch.stack([a.cos(), a.sin()], -1).float()


def angles(positions: torch.Tensor, rot: Rotary) -> torch.Tensor:
    """``positions [...]`` (below 0 = padding, taken as 0) -> ``[..., dims / 2, 2]`` fp32: cosine and sine of every pair's angle."""
    if not L.use_cuda(positions):
        return angles_reference(positions, rot)
    p = positions.to(torch.int32).contiguous()
    f = _frequencies(rot, p.device)
    out = torch.empty(*p.shape, rot.dims // 2, 2, dtype=torch.float32, device=p.device)
    L.check(L.load().dewb_rotary_angles(L.ptr(p), L.ptr(f), L.ptr(out), c_ll(p.numel()), c_int(rot.dims // 2), L.stream_ptr()), "rotary_angles")
    L.count_launches()
    return out


def turn(x: torch.Tensor, table: Optional[torch.Tensor], rot: Rotary) -> torch.Tensor:
    """``x [..., heads, width]`` in fp32 with its first ``dims`` dimensions turned by ``table [..., dims / 2, 2]``."""
    x = x.float()
    cos, sin = table[..., None, :, 0], table[..., None, :, 1]
    part, rest = x[..., :rot.dims], x[..., rot.dims:]
    if rot.interleaved:
        u, v = part[..., 0::2], part[..., 1::2]
        out = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
    else:
        u, v = part.chunk(2, -1)
        out = torch.cat([u * cos - v * sin, v * cos + u * sin], -1)
    return torch.cat([out, rest], -1)
