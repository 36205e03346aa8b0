"""Latent attention in generation (``csrc/kernels/latent_attention.cu``), each operation with its plain PyTorch form.

A layer's input projection is ``[query latent | latent | key part | gate]``; a token leaves ``[normed latent | rotated key part]`` in its page, one row
for all heads.  Two forms of the same attention:

* in the latents' space (``absorb`` -> ``attend`` -> ``expand``): the key up-projection moves to the queries and the value up-projection behind the
  sum, so a decode step reads one row per cached token for all heads;
* in full width (``rotate`` -> the layer's up-projection of the latents -> flash attention over two-part keys): prompts, and their later portions
  after ``gather``.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import NamedTuple, Optional, Tuple

import torch

from . import library as L
from . import paged as P
from .rotary import Rotary, turn

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float
MAX_WIDTH, MAX_RANK = 584, 512          # what the tensor-core kernel against the latents takes; past them, the general paged kernel


@dataclass(frozen=True)
class Latent:
    """The shape of one latent attention layer: heads, their unrotated and rotated query / key widths, their value width, the latents' widths
    (``q_rank`` 0: queries without one), and the rotation of the rotated part."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    q_rank: int
    rotary: Rotary

    def __post_init__(self):
        if self.rotary.dims > self.rot_dim:
            raise ValueError(f"a rotation of {self.rotary.dims} dimensions does not fit the rotated part of {self.rot_dim}")

    @property
    def width(self) -> int:
        """A query / key head."""
        return self.dim + self.rot_dim

    @property
    def row(self) -> int:
        """What a token leaves."""
        return self.rank + self.rot_dim

    def split_up(self, up: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """The up-projection ``[heads * (dim + vdim), rank]`` as keys ``[heads, dim, rank]`` and values ``[heads, vdim, rank]``."""
        w = up.view(self.heads, self.dim + self.vdim, self.rank)
        return w[:, :self.dim], w[:, self.dim:]


class Rows(NamedTuple):
    """What a call's tokens left: latents ``[R, S, rank]`` and rotated key parts ``[R, S, rot_dim]``."""
    c: torch.Tensor
    key: torch.Tensor


def prepare_reference(z, lat: Latent, qw, cw, eps: float, table) -> Tuple[Optional[torch.Tensor], Rows]:
    """``z [R, S, *]`` -> the normed query latent (None without one) and the tokens' rows, in ``z``'s dtype."""
    q, c, k = z[..., :lat.q_rank + lat.row].split([lat.q_rank, lat.rank, lat.rot_dim], -1)
    q = P.rms_norm_fp32(q, qw, eps).to(z.dtype) if lat.q_rank else None
    return q, Rows(P.rms_norm_fp32(c, cw, eps).to(z.dtype), turn(k.unsqueeze(-2), table, lat.rotary).squeeze(-2).to(z.dtype))


def rows(z: torch.Tensor, lat: Latent, qw, cw, eps: float, table: torch.Tensor, positions: torch.Tensor, pages: P.Pages) -> Tuple[Optional[torch.Tensor], Rows]:
    """``prepare_reference`` with the rows of the live positions written to ``pages.k [*, page_size, 1, W]``."""
    R, S = positions.shape
    W = pages.k.shape[-1]
    if L.use_cuda(z):
        z = z.contiguous()
        made = lambda n: torch.empty(R, S, n, dtype=z.dtype, device=z.device)
        cq, out = made(lat.q_rank), Rows(made(lat.rank), made(lat.rot_dim))
        qw, cw = (None if w is None else w.detach().to(z.dtype).contiguous() for w in (qw, cw))
        L.check(L.load().dewb_latent_rows(L.ptr(z), c_ll(z.shape[-1]), L.ptr(qw), L.ptr(cw), c_float(eps), L.ptr(table), c_int(lat.rotary.dims),
                                          c_int(int(lat.rotary.interleaved)), L.ptr(positions), c_int(R), c_int(S), c_int(lat.q_rank), c_int(lat.rank),
                                          c_int(lat.rot_dim), c_int(W), L.ptr(cq), L.ptr(out.c), L.ptr(out.key), L.ptr(pages.k), L.ptr(pages.table),
                                          c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids), c_int(int(z.dtype == torch.float32)),
                                          L.stream_ptr()), "latent_rows")
        L.count_launches()
        return (cq if lat.q_rank else None), out
    cq, out = prepare_reference(z, lat, qw, cw, eps, table)
    slots, live = P._slots(pages, positions), positions >= 0
    row = torch.nn.functional.pad(torch.cat(out, -1), (0, W - lat.row))
    pages.k.view(-1, W)[slots[live]] = row[live].to(pages.k.dtype)
    return cq, out


def rotate(q: torch.Tensor, lat: Latent, table: torch.Tensor) -> torch.Tensor:
    """``q [R, S, H, width]`` with every head's rotated part turned; on a GPU in place."""
    if not L.use_cuda(q):
        return torch.cat([q[..., :lat.dim], turn(q[..., lat.dim:], table, lat.rotary).to(q.dtype)], -1)
    q = q.contiguous()
    L.check(L.load().dewb_rotate_tail(L.ptr(q), L.ptr(table), c_ll(q.numel() // (lat.heads * lat.width)), c_int(lat.heads), c_int(lat.width), c_int(lat.dim),
                                      c_int(lat.rotary.dims), c_int(int(lat.rotary.interleaved)), c_int(int(q.dtype == torch.float32)), L.stream_ptr()), "rotate_tail")
    L.count_launches()
    return q


def _product(a: torch.Tensor, w: torch.Tensor, trans: bool, out: torch.Tensor, n: int, k: int, gate=None, lat: Optional[Latent] = None, table=None, pad: int = 0):
    """``out [T, H, :n] = a [T, H, :k]`` times ``w [H, n, k]`` (``trans``: ``[H, k, n]``, both unit stride along the last axis)."""
    T, H = a.shape[:2]
    w = w.to(a.dtype)
    L.check(L.load().dewb_head_product(L.ptr(a), c_ll(a.stride(0)), c_ll(a.stride(1)), L.ptr(w), c_ll(w.stride(0)), c_ll(w.stride(1)), c_int(int(trans)), L.ptr(gate),
                                       c_ll(0 if gate is None else gate.stride(0)), L.ptr(out), c_ll(out.stride(0)), c_ll(out.stride(1)), c_int(T), c_int(H),
                                       c_int(n), c_int(k), L.ptr(table), c_int(0 if lat is None else lat.rot_dim), c_int(pad),
                                       c_int(0 if lat is None else lat.rotary.dims), c_int(int(lat is not None and lat.rotary.interleaved)),
                                       c_int(int(a.dtype == torch.float32)), L.stream_ptr()), "head_product")
    L.count_launches()
    return out


def absorb(q: torch.Tensor, up: torch.Tensor, lat: Latent, table: torch.Tensor, W: int) -> torch.Tensor:
    """``q [R, S, H, width]`` -> queries against the rows in the pages, ``[R, S, H, W]``."""
    R, S, H, _ = q.shape
    wk, _ = lat.split_up(up.detach())
    if L.use_cuda(q):
        q = q.contiguous()
        out = torch.empty(R, S, H, W, dtype=q.dtype, device=q.device)
        _product(q.view(R * S, H, lat.width), wk, True, out.view(R * S, H, W), lat.rank, lat.dim, None, lat, table, W - lat.rank)
        return out
    c = torch.einsum("rshd,hdl->rshl", q[..., :lat.dim].float(), wk.float())
    turned = turn(q[..., lat.dim:], table, lat.rotary)
    return torch.nn.functional.pad(torch.cat([c, turned], -1), (0, W - lat.row)).to(q.dtype)


def gate_reference(o: torch.Tensor, gate: Optional[torch.Tensor]) -> torch.Tensor:
    return o if gate is None else (o.float() * torch.sigmoid(gate.float())).to(o.dtype)


def expand(o: torch.Tensor, up: torch.Tensor, lat: Latent, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Sums of latents ``o [R, S, H, rank]`` -> the heads' values ``[R, S, H * vdim]``, times the sigmoid of ``gate`` (columns of the projection)."""
    R, S, H, _ = o.shape
    _, wv = lat.split_up(up.detach())
    if L.use_cuda(o):
        o = o.contiguous()
        out = torch.empty(R, S, H * lat.vdim, dtype=o.dtype, device=o.device)
        g = None if gate is None else flat_gate(gate)
        _product(o.view(R * S, H, lat.rank), wv, False, out.view(R * S, H, lat.vdim), lat.vdim, lat.rank, g)
        return out
    v = torch.einsum("rshl,hvl->rshv", o.float(), wv.float()).to(o.dtype)
    return gate_reference(v.reshape(R, S, H * lat.vdim), gate)


def flat_gate(gate: torch.Tensor) -> torch.Tensor:
    """``[R, S, n]`` (columns of a wider tensor will do) as ``[R * S, n]`` with one row stride."""
    if gate.stride(-1) != 1 or (gate.shape[0] > 1 and gate.stride(0) != gate.shape[1] * gate.stride(1)):
        gate = gate.contiguous()
    return gate.as_strided((gate.shape[0] * gate.shape[1], gate.shape[2]), (gate.stride(1), 1))


def attend_kernel_ok(q: torch.Tensor, lat: Latent, W: int) -> bool:
    return q.dtype == torch.bfloat16 and W % 16 == 8 and W <= MAX_WIDTH and lat.rank <= MAX_RANK


def attend(q: torch.Tensor, lat: Latent, positions: torch.Tensor, pages: P.Pages, scale: float, longest: int, scratch=None,
           kernel: Optional[str] = None) -> torch.Tensor:
    """``q [R, S, H, W]`` against the rows' latents -> sums of latents ``[R, S, H, rank]``.  ``longest``: keys a row may hold; ``scratch(n, width)`` lends
    fp32 buffers for the partial sums.  ``kernel`` forces ``mma`` or ``general``."""
    R, S, H, W = q.shape
    if not L.use_cuda(q) or (kernel or ("mma" if attend_kernel_ok(q, lat, W) else "general")) == "general":
        return P.paged_attend(q, P.Heads(H, 1, lat.row, lat.rank), positions, pages, scale, kernel="general")
    q = q.contiguous()
    out = torch.empty(R, S, H, lat.rank, dtype=q.dtype, device=q.device)
    wide = S * H > 16
    blocks, tiles = R * -(-S * H // (32 if wide else 16)), -(-longest // 32)
    splits = max(1, min(148 // max(blocks, 1), tiles // 4, 32))      # one CTA an SM
    pm = pl = pa = None
    if splits > 1:
        n = R * S * H * splits
        pm, pl, pa = (scratch or fresh_scratch(q.device))(n, lat.rank)
    L.check(L.load().dewb_latent_attend(L.ptr(q), L.ptr(pages.k), L.ptr(positions), c_int(R), c_int(S), c_int(H), c_int(W), c_int(lat.rank), c_float(scale),
                                        c_int(splits), c_int(int(wide)), L.ptr(pm), L.ptr(pl), L.ptr(pa), L.ptr(out), L.ptr(pages.table),
                                        c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids), L.ptr(L.status(q.device)), L.stream_ptr()),
            "latent_attend")
    L.count_launches(1 + int(splits > 1))
    return out


def fresh_scratch(device):
    make = lambda n: torch.empty(n, dtype=torch.float32, device=device)
    return lambda n, width: (make(n), make(n), make(n * width))


def gather(lat: Latent, lengths: torch.Tensor, total: int, pages: P.Pages) -> Rows:
    """The first ``total`` tokens of every row as dense rows, zeros past ``lengths [R]``."""
    R, pool = lengths.numel(), pages.k
    out = Rows(*(torch.empty(R, total, n, dtype=pool.dtype, device=pool.device) for n in (lat.rank, lat.rot_dim)))
    L.check(L.load().dewb_latent_gather(L.ptr(pool), L.ptr(lengths), c_int(R), c_int(total), c_int(lat.rank), c_int(lat.rot_dim), c_int(pool.shape[-1]),
                                        L.ptr(out.c), L.ptr(out.key), L.ptr(pages.table), c_int(pages.page_size), c_int(pages.table.shape[1]),
                                        L.ptr(pages.row_ids), c_int(int(pool.dtype == torch.float32)), L.stream_ptr()), "latent_gather")
    L.count_launches()
    return out


def flash_ok(q: torch.Tensor, lat: Latent) -> bool:
    """Whether the tcgen05 kernel takes the full-width form."""
    sub = -(-lat.dim // 64) + -(-lat.rot_dim // 64)
    return (q.dtype == torch.bfloat16 and q.shape[1] % 128 == 0 and lat.dim % 8 == 0 and lat.rot_dim % 8 == 0 and lat.vdim % 8 == 0 and lat.rank % 8 == 0
            and sub <= 3 and lat.vdim <= 128)


def flash(q: torch.Tensor, made: Rows, up: torch.Tensor, lat: Latent, scale: float, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rotated queries ``q [R, S, H, width]`` against the rows ``made [R, T, *]`` in full width, query i seeing the keys up to ``i + T - S`` ->
    ``[R, S, H * vdim]``, times the sigmoid of ``gate``."""
    from .functional import linear
    R, S, H, _ = q.shape
    T = made.c.shape[1]
    kv = linear(made.c, up).view(R, T, H, lat.dim + lat.vdim)
    k, v = kv[..., :lat.dim], kv[..., lat.dim:]
    out = torch.empty(R, S, H * lat.vdim, dtype=q.dtype, device=q.device)
    g = None if gate is None else flat_gate(gate)
    if g is not None and (g.stride(0) % 8 or g.data_ptr() % 16):
        g = g.contiguous()
    three = lambda t: (c_ll(t.stride(0)), c_ll(t.stride(1)), c_ll(t.stride(2)))
    L.check(L.load().dewb_flash_fwd_parts(L.ptr(q), L.ptr(k), L.ptr(made.key), L.ptr(v), L.ptr(g), c_ll(0 if g is None else g.stride(0)), L.ptr(out), c_int(R),
                                          c_int(S), c_int(T), c_int(H), c_int(lat.dim), c_int(lat.rot_dim), c_int(lat.vdim), *three(q), *three(k),
                                          c_ll(made.key.stride(0)), c_ll(made.key.stride(1)), *three(v), c_float(scale), L.ptr(L.status(q.device)),
                                          L.stream_ptr()), "flash_fwd_parts")
    L.count_launches()
    return out
