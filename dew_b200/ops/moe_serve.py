"""Mixture-of-experts feed-forward outside training (``csrc/kernels/moe_serve.cu``): selection, expert-sorted rows, grouped products and the
weighted sum with the shared expert, without statistics, saved state or host synchronisation (a decode step that runs it can be captured into
a CUDA graph).  ``select_reference`` is the selection's plain PyTorch form.
"""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional, Tuple

import torch

from . import grouped as G
from . import library as L

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float
MAX_EXPERTS, MAX_TOP = 1024, 32
SCORES = ("softmax", "sigmoid", "top_softmax")
ROUTER_TOKENS = 512          # up to here the router's logits are formed token by token; past it, by a tensor-core product


class Selection(NamedTuple):
    """How a router chooses: ``top`` of ``experts``; with ``groups`` > 1 only within the token's best ``keep`` groups (by the sum of their ``best``,
    one or two, best choice scores), the others' choice scores becoming ``fill``; ``norm`` divides the weights by their sum.  ``score``: ``softmax`` or ``sigmoid``
    of the logits, or ``top_softmax``: the choice runs on the logits, and the weights are the softmax over the chosen ones alone."""
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    fill: float = 0.0
    score: str = "softmax"
    norm: bool = True
    scaling: float = 1.0
    best: int = 2


def choice_scores(scores: torch.Tensor, bias: Optional[torch.Tensor], s: Selection) -> torch.Tensor:
    """``scores [T, E]`` -> what the top-k runs on: the bias added, experts outside the kept groups filled."""
    select = scores if bias is None else scores + bias
    if s.groups > 1:
        T, E = select.shape
        per = E // s.groups
        best = select.view(T, s.groups, per).topk(min(s.best, per), -1).values.sum(-1)
        keep = torch.zeros_like(best).scatter_(1, best.topk(s.keep, -1).indices, 1.0).bool()
        select = select.masked_fill(~keep[:, :, None].expand(T, s.groups, per).reshape(T, E), s.fill)
    return select


def select_reference(logits: torch.Tensor, bias: Optional[torch.Tensor], s: Selection) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """fp32 ``logits [T, E]`` -> (weights ``[T, k]``, ids ``[T, k]``, scores ``[T, E]``)."""
    if s.score not in SCORES:
        raise ValueError(f"unknown router score {s.score!r}; known: {', '.join(SCORES)}")
    if s.score == "top_softmax":
        ids = torch.topk(choice_scores(logits, bias, s), s.top, dim=-1).indices
        return torch.softmax(logits.gather(-1, ids), -1) * s.scaling, ids, torch.softmax(logits, -1)
    scores = torch.softmax(logits, -1) if s.score == "softmax" else torch.sigmoid(logits)
    ids = torch.topk(choice_scores(scores, bias, s), s.top, dim=-1).indices
    w = scores.gather(-1, ids)
    if s.norm:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return w * s.scaling, ids, scores


class Split(NamedTuple):
    """A router's fp32 weights as bf16 rows: the rounded weights, and (where the rounding dropped anything) what it dropped below them."""
    rows: torch.Tensor
    exact: bool


def split_weights(w: torch.Tensor) -> Split:
    w = w.detach().float()
    big = w.to(torch.bfloat16)
    rest = (w - big.float()).to(torch.bfloat16)
    exact = not bool(rest.any())
    pad = -w.shape[0] % 8                                       # (the second half starts on a multiple of eight columns of the logits)
    return Split(big if exact else torch.cat([torch.nn.functional.pad(big, (0, 0, 0, pad)), rest]).contiguous(), exact)


def usable(x2: torch.Tensor, s: Selection) -> bool:
    return s.experts <= MAX_EXPERTS and s.top <= MAX_TOP and x2.dtype in (torch.bfloat16, torch.float32) and L.use_cuda(x2)


class Routed(NamedTuple):
    weights: torch.Tensor        # [T, k] fp32
    ids: torch.Tensor            # [T, k] int32, -1: padding
    rank: torch.Tensor           # [T, k] int32: place among the expert's rows
    counts: torch.Tensor         # [E] int32


def route(x2: torch.Tensor, weight: torch.Tensor, split: Optional[Split], bias: Optional[torch.Tensor], s: Selection,
          positions: Optional[torch.Tensor] = None, kernel: Optional[str] = None, logit_bias: Optional[torch.Tensor] = None) -> Routed:
    """``x2 [T, d]``, the router's ``weight [E, d]`` (``split``: its bf16 rows, for a bf16 ``x2``), ``bias`` of the choice, ``logit_bias`` of the logits.  ``kernel`` forces ``rows`` (logits token by
    token) or ``product`` (a tensor-core product first)."""
    T, d = x2.shape
    E, k, dev = s.experts, s.top, x2.device
    out = Routed(torch.empty(T, k, dtype=torch.float32, device=dev), torch.empty(T, k, dtype=torch.int32, device=dev),
                 torch.empty(T, k, dtype=torch.int32, device=dev), torch.zeros(E, dtype=torch.int32, device=dev))
    x2, lib = x2.contiguous(), L.load()
    b, lb = (None if t is None else t.detach().float().contiguous() for t in (bias, logit_bias))
    if positions is not None and positions.numel() != T:
        raise ValueError(f"{positions.numel()} positions for {T} tokens")
    tail = (c_int(E), c_int(k), c_int(s.groups), c_int(s.keep), c_int(s.best), c_float(s.fill), c_int(SCORES.index(s.score)), c_int(int(s.norm)), c_float(s.scaling),
            L.ptr(out.weights), L.ptr(out.ids), L.ptr(out.rank), L.ptr(out.counts))
    if (kernel or ("product" if T > ROUTER_TOKENS and x2.dtype == torch.bfloat16 and split is not None and d % 8 == 0 else "rows")) == "product":
        from .functional import gemm
        n = split.rows.shape[0]
        ld = (n + 7) // 8 * 8
        logits = torch.empty(T, ld, dtype=torch.float32, device=dev)
        gemm(x2, split.rows, out=logits[:, :n], kernel="sm100_tcgen05")
        L.check(lib.dewb_moe_select(L.ptr(logits), c_ll(ld), c_int(0 if split.exact else n - E), L.ptr(b), L.ptr(lb), L.ptr(positions), c_int(T), *tail, L.stream_ptr()),
                "moe_select")
        L.count_launches()
        return out
    w = split.rows if split is not None and split.exact and x2.dtype == torch.bfloat16 else weight.detach().float()
    w = w.contiguous()
    L.check(lib.dewb_moe_router(L.ptr(x2), L.ptr(w), L.ptr(b), L.ptr(lb), L.ptr(positions), c_int(T), c_int(d), *tail, c_int(int(x2.dtype == torch.float32)),
                                c_int(int(w.dtype == torch.float32)), L.stream_ptr()), "moe_router")
    L.count_launches()
    return out


class Sorted(NamedTuple):
    rows: torch.Tensor           # [tiles * 128, d]; rows no token has are left as they were
    place: torch.Tensor          # [T, k] int32 row of each choice, -1: padding
    tile_group: torch.Tensor     # [tiles] int32
    offsets: torch.Tensor        # [E + 1] int32
    counts: torch.Tensor
    gate: Optional[torch.Tensor]  # [T] fp32: the shared expert's


def gather(x2: torch.Tensor, r: Routed, gate_weight: Optional[torch.Tensor] = None) -> Sorted:
    T, d = x2.shape
    k, E, dev = r.ids.shape[1], r.counts.numel(), x2.device
    tiles = G.padded_rows(T * k, min(E, T * k)) // G.BLOCK
    x2 = x2.contiguous()
    gw = None if gate_weight is None else gate_weight.detach().to(x2.dtype).reshape(-1).contiguous()
    ints = dict(dtype=torch.int32, device=dev)
    out = Sorted(torch.empty(tiles * G.BLOCK, d, dtype=x2.dtype, device=dev), torch.empty(T, k, **ints), torch.empty(tiles, **ints), torch.empty(E + 1, **ints),
                 r.counts, None if gw is None else torch.empty(T, dtype=torch.float32, device=dev))
    L.check(L.load().dewb_moe_gather(L.ptr(x2), L.ptr(r.ids), L.ptr(r.rank), L.ptr(r.counts), L.ptr(gw), L.ptr(out.rows), L.ptr(out.place), L.ptr(out.tile_group),
                                     L.ptr(out.offsets), L.ptr(out.gate), c_int(T), c_int(d), c_int(E), c_int(k), c_int(tiles),
                                     c_int(int(x2.dtype == torch.float32)), L.stream_ptr()), "moe_gather")
    L.count_launches()
    return out


def product(a: torch.Tensor, w: torch.Tensor, s: Sorted, kernel: Optional[str] = None) -> torch.Tensor:
    """``a [rows, K] @ w[expert of the row]^T`` with ``w [E, N, K]``: tcgen05 for bf16 rows of whole 16-byte pieces, else the CUDA cores.
    ``kernel`` forces ``tensor`` or ``general``."""
    E, N, K = w.shape
    tiles = s.tile_group.numel()
    out = torch.empty(a.shape[0], N, dtype=a.dtype, device=a.device)
    if (kernel or ("tensor" if a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and K % 8 == 0 else "general")) == "tensor":
        return G.gmm_forward(a, w.detach(), G.GroupLayout(None, s.counts, s.offsets, s.tile_group, a.shape[0]), out=out)
    w = w.detach().to(a.dtype).contiguous()
    L.check(L.load().dewb_moe_gemm(L.ptr(a), L.ptr(w), L.ptr(out), L.ptr(s.tile_group), L.ptr(s.offsets), L.ptr(s.counts), c_int(tiles), c_int(N), c_int(K),
                                   c_int(int(a.dtype == torch.float32)), L.stream_ptr()), "moe_gemm")
    L.count_launches()
    return out


def glu(gu: torch.Tensor, s: Sorted) -> torch.Tensor:
    """``silu(gate) * up`` of the rows in use, ``[rows, 2 F] -> [rows, F]``."""
    F = gu.shape[1] // 2
    out = torch.empty(gu.shape[0], F, dtype=gu.dtype, device=gu.device)
    L.check(L.load().dewb_moe_glu(L.ptr(gu), L.ptr(out), L.ptr(s.tile_group), L.ptr(s.offsets), L.ptr(s.counts), c_int(s.tile_group.numel()), c_int(F),
                                  c_int(int(gu.dtype == torch.float32)), L.stream_ptr()), "moe_glu")
    L.count_launches()
    return out


def combine(y: torch.Tensor, r: Routed, s: Sorted, shared: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[t] = sum_j weights[t, j] y[place[t, j]] (+ gate[t] shared[t])`` in fp32 -> ``[T, d]``."""
    T, k = r.ids.shape
    d = y.shape[1]
    out = torch.empty(T, d, dtype=y.dtype, device=y.device)
    shared = None if shared is None else shared.contiguous()
    L.check(L.load().dewb_moe_combine(L.ptr(y), L.ptr(r.weights), L.ptr(s.place), L.ptr(shared), L.ptr(s.gate), L.ptr(out), c_int(T), c_int(d), c_int(k),
                                      c_int(int(y.dtype == torch.float32)), L.stream_ptr()), "moe_combine")
    L.count_launches()
    return out
