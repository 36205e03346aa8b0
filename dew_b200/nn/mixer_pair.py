"""Two mixers side by side over one input, whose outputs are added with a factor each."""
from __future__ import annotations

from typing import Tuple

import torch
import torch.nn as nn


class MixerPair(nn.Module):
    """``left_scale * left(x) + right_scale * right(x)``.  In a cache the left mixer has the layer run's slot and the right one the slot beside it."""

    def __init__(self, left: nn.Module, right: nn.Module, left_rotary: bool, right_rotary: bool, left_scale: float = 1.0, right_scale: float = 1.0):
        super().__init__()
        self.left, self.right = left, right
        self.rotary = (left_rotary, right_rotary)          # whether a mixer is called with rotary tables
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)

    def cache_slot(self):
        from dataclasses import replace
        return replace(self.left.cache_slot(), beside=self.right.cache_slot())

    def branches(self, x, segment_ids=None, cache=None, layer: int = 0, positions=None) -> Tuple[torch.Tensor, torch.Tensor]:
        """The two outputs without their factors."""
        out = []
        cached = getattr(cache, "beside", None) is not None
        for mixer, rotary, slot in ((self.left, self.rotary[0], layer), (self.right, self.rotary[1], cache.beside[layer] if cached else layer)):
            if rotary:
                out.append(mixer(x, None, None, positions, segment_ids, cache, slot))
            else:
                out.append(mixer(x, segment_ids=segment_ids, cache=cache if cached else None, layer=slot, positions=positions))
        return out[0], out[1]

    def forward(self, x, segment_ids=None, cache=None, layer: int = 0, positions=None) -> torch.Tensor:
        a, b = self.branches(x, segment_ids, cache, layer, positions)
        return (self.left_scale * a.float() + self.right_scale * b.float()).to(x.dtype)
