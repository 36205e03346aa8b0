"""Attention of a call's tokens against a paged cache of any head widths (``csrc/kernels/paged_attention.cu``) and the projection
epilogue in front of it (norm over all heads, query temperature, append), each with its plain PyTorch form."""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional

import torch

from . import library as L

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class Heads(NamedTuple):
    """The shape of one attention layer: query heads, key / value heads, key width, value width."""
    q: int
    kv: int
    dk: int
    dv: int

    @property
    def packed(self) -> int:
        return (self.q + self.kv) * self.dk + self.kv * self.dv


class Pages(NamedTuple):
    """A layer's page pools and where a call's rows live in them."""
    k: torch.Tensor                       # [pages, page_size, kv heads, width]
    v: torch.Tensor
    table: torch.Tensor                   # [store rows, max_pages] int32
    page_size: int
    row_ids: Optional[torch.Tensor]       # int32 store row of each call row (None: the same)


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """``1 + coef ln(floor((p + 1) / every) + 1)`` in fp32."""
    return 1.0 + coef * torch.log(((positions + 1) // every + 1).float())


def rms_norm_fp32(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    if w is None:
        return x.float()
    xf = x.float()
    return xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def prepare_reference(qkv, heads: Heads, qw, kw, eps: float, temperature, positions):
    """``q [R, S, H, dk]``, ``k [R, S, G, dk]``, ``v [R, S, G, dv]`` after the norms and the temperature, in the projection's dtype."""
    R, S, _ = qkv.shape
    q, k, v = qkv.split([heads.q * heads.dk, heads.kv * heads.dk, heads.kv * heads.dv], -1)
    q, k = rms_norm_fp32(q, qw, eps), rms_norm_fp32(k, kw, eps)
    if temperature is not None:
        q = q * query_temperature(positions.clamp_min(0), temperature[0], temperature[1]).unsqueeze(-1)
    return (q.to(qkv.dtype).view(R, S, heads.q, heads.dk), k.to(qkv.dtype).view(R, S, heads.kv, heads.dk), v.reshape(R, S, heads.kv, heads.dv))


def _slots(pages: Pages, positions: torch.Tensor) -> torch.Tensor:
    R = positions.shape[0]
    rows = torch.arange(R, device=positions.device) if pages.row_ids is None else pages.row_ids.long()
    p = positions.clamp_min(0).long()
    return pages.table[rows[:, None], p // pages.page_size].long() * pages.page_size + p % pages.page_size


def qk_norm_append(qkv, heads: Heads, qw, kw, eps: float, temperature, positions, pages: Pages) -> torch.Tensor:
    """-> ``[R, S, H + 2 G, D]`` (normalised queries and keys, values; every head padded with zeros to the pool's width), with the keys and
    values of the live positions written to the pools.  ``positions`` int32 ``[R, S]``, below 0 = padding."""
    R, S, _ = qkv.shape
    D = pages.k.shape[-1]
    if L.use_cuda(qkv):
        qkv = qkv.contiguous()
        qw, kw = (None if w is None else w.detach().to(qkv.dtype).contiguous() for w in (qw, kw))
        packed = torch.empty(R, S, heads.q + 2 * heads.kv, D, dtype=qkv.dtype, device=qkv.device)
        coef, every = temperature if temperature is not None else (0.0, 0)
        L.check(L.load().dewb_qk_norm_append(L.ptr(qkv), L.ptr(qw), L.ptr(kw), c_float(eps), c_float(coef), c_int(every), L.ptr(positions), c_int(R),
                                             c_int(S), c_int(heads.q), c_int(heads.kv), c_int(heads.dk), c_int(heads.dv), c_int(D), L.ptr(packed),
                                             L.ptr(pages.k), L.ptr(pages.v), L.ptr(pages.table), c_int(pages.page_size), c_int(pages.table.shape[1]),
                                             L.ptr(pages.row_ids), c_int(int(qkv.dtype == torch.float32)), L.stream_ptr()), "qk_norm_append")
        L.count_launches()
        return packed
    q, k, v = prepare_reference(qkv, heads, qw, kw, eps, temperature, positions)
    pad = lambda t: torch.nn.functional.pad(t, (0, D - t.shape[-1]))
    q, k, v = pad(q), pad(k), pad(v)
    slots, live = _slots(pages, positions), positions >= 0
    for pool, t in ((pages.k, k), (pages.v, v)):
        pool.view(-1, heads.kv, D)[slots[live]] = t[live].to(pool.dtype)
    return torch.cat([q, k, v], 2)


def paged_attend_reference(q, heads: Heads, positions, pages: Pages, scale: float) -> torch.Tensor:
    R, S = positions.shape
    D = pages.k.shape[-1]
    n = int(positions.max()) + 1
    if n <= 0:
        return q.new_zeros(R, S, heads.q, heads.dv)
    slots = _slots(pages, torch.arange(n, device=q.device)[None].expand(R, n))
    kc = pages.k.view(-1, heads.kv, D)[slots].float().repeat_interleave(heads.q // heads.kv, 2)          # [R, n, H, D]
    vc = pages.v.view(-1, heads.kv, D)[slots][..., :heads.dv].float().repeat_interleave(heads.q // heads.kv, 2)
    seen = torch.arange(n, device=q.device)[None, None] <= positions[..., None]                          # [R, S, n]
    # what the pool holds beyond a row's own tokens is another row's, or nothing: it must not reach the sums
    own = (torch.arange(n, device=q.device)[None] <= positions.amax(1, keepdim=True))[..., None, None]
    kc, vc = torch.where(own, kc, torch.zeros_like(kc)), torch.where(own, vc, torch.zeros_like(vc))
    s = torch.einsum("rshd,rnhd->rhsn", q[..., :D].float(), kc) * scale
    p = torch.nan_to_num(torch.softmax(s.masked_fill(~seen[:, None], float("-inf")), -1))
    return torch.einsum("rhsn,rnhd->rshd", p, vc).to(q.dtype)


def paged_attend(q: torch.Tensor, heads: Heads, positions: torch.Tensor, pages: Pages, scale: float, kernel: Optional[str] = None) -> torch.Tensor:
    """``q [R, S, H, D]`` (a view into the packed tensor will do: unit stride in a head, heads next to each other) -> ``[R, S, H, dv]``.
    ``kernel`` forces ``mma`` (bf16 pools of 64, 128, 256) or ``general``."""
    if not L.use_cuda(q):
        return paged_attend_reference(q, heads, positions, pages, scale)
    R, S, H, D = q.shape
    if q.stride(3) != 1 or q.stride(2) != D or (R > 1 and q.stride(0) != S * q.stride(1)):
        q = q.contiguous()
    out = torch.empty(R, S, H, heads.dv, dtype=q.dtype, device=q.device)
    if (kernel or ("mma" if q.dtype == torch.bfloat16 and D in (64, 128, 256) else "general")) == "mma":
        L.check(L.load().dewb_paged_attend_mma(L.ptr(q), c_ll(q.stride(1)), L.ptr(pages.k), L.ptr(pages.v), L.ptr(positions), c_int(R), c_int(S), c_int(H),
                                               c_int(heads.kv), c_int(heads.dv), c_int(D), c_float(scale), L.ptr(out), L.ptr(pages.table),
                                               c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids), L.stream_ptr()), "paged_attend_mma")
        L.count_launches()
        return out
    L.check(L.load().dewb_paged_attend(L.ptr(q), c_ll(q.stride(1)), L.ptr(pages.k), L.ptr(pages.v), L.ptr(positions), c_int(R), c_int(S), c_int(H),
                                       c_int(heads.kv), c_int(heads.dk), c_int(heads.dv), c_int(D), c_float(scale), L.ptr(out), L.ptr(pages.table),
                                       c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids),
                                       c_int(int(q.dtype == torch.float32)), L.stream_ptr()), "paged_attend")
    L.count_launches()
    return out
