"""Attention of a call's tokens against a paged cache of any head widths (``csrc/kernels/paged_attention.cu``), the projection epilogue in
front of it (bias, norm over all heads or per head, rotation, query temperature, append) and the head gate behind it, each with its plain PyTorch
form."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Iterator, NamedTuple, Optional

import torch

from . import library as L
from . import rotary as rotary_ops

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float


@dataclass(frozen=True)
class Heads:
    """The shape of one attention layer: query heads, key / value heads, key width, value width; ``own``: it projects keys and values of its
    own (else it reads another layer's); ``gated``: its projection ends in one gate per query head."""
    q: int
    kv: int
    dk: int
    dv: int
    own: bool = True
    gated: bool = False

    def __iter__(self) -> Iterator[int]:
        """The four sizes."""
        return iter((self.q, self.kv, self.dk, self.dv))

    @property
    def packed(self) -> int:
        """Columns of the heads in the projection."""
        return self.q * self.dk + (self.kv * (self.dk + self.dv) if self.own else 0)

    @property
    def row(self) -> int:
        """Columns of the projection."""
        return self.packed + (self.q if self.gated else 0)


class Visible(NamedTuple):
    """What a layer's attention adds to the causal softmax: a query sees no key from before the start of its ``chunk`` of positions; with a ``window``
    it sees that many keys (its own included) and the row's first ``keep``; scores are multiplied by ``gain`` (fp32, one per query head) and become
    ``softcap tanh(score / softcap)``; ``sinks`` (fp32, one per query head) join the denominator only.  With ``sigmoid`` (fp32, one per query head) there is
    no softmax: a visible key weighs ``sigmoid(score + sigmoid[head])``."""
    chunk: Optional[int] = None
    sinks: Optional[torch.Tensor] = None
    window: Optional[int] = None
    keep: int = 0
    softcap: float = 0.0
    gain: Optional[torch.Tensor] = None
    sigmoid: Optional[torch.Tensor] = None


PLAIN = Visible()


class Pages(NamedTuple):
    """A layer's page pools and where a call's rows live in them."""
    k: torch.Tensor                       # [pages, page_size, kv heads, width]
    v: torch.Tensor
    table: torch.Tensor                   # [store rows, max_pages] int32
    page_size: int
    row_ids: Optional[torch.Tensor]       # int32 store row of each call row (None: the same)


class Turned(NamedTuple):
    """A call's rotation of the query and key heads: ``table`` of ``rotary.angles``."""
    rot: rotary_ops.Rotary
    table: torch.Tensor


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """``1 + coef ln(floor((p + 1) / every) + 1)`` in fp32."""
    return 1.0 + coef * torch.log(((positions + 1) // every + 1).float())


def rms_norm_fp32(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    if w is None:
        return x.float()
    xf = x.float()
    return xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def per_head(heads: Heads, qw, kw) -> bool:
    """Whether the norms' weights are of one head (shared by all) rather than of all heads at once."""
    return (qw is not None and qw.numel() != heads.q * heads.dk) or (kw is not None and kw.numel() != heads.kv * heads.dk)


def prepare_reference(qkv, heads: Heads, qw, kw, eps: float, temperature, positions, bias=None, turned: Optional[Turned] = None, unit: bool = False):
    """``q [R, S, H, dk]``, ``k [R, S, G, dk]``, ``v [R, S, G, dv]`` after the bias, the norms, the rotation, (with ``unit``) the division of every head by
    its root mean square, and the temperature, in the projection's dtype (keys and values None for a layer without its own)."""
    R, S, _ = qkv.shape
    one = per_head(heads, qw, kw)

    def norm(t, n, w):
        t = t.reshape(R, S, n, heads.dk) if one else t
        t = rms_norm_fp32(t, w, eps).reshape(R, S, n, heads.dk)
        if turned is not None:
            t = rotary_ops.turn(t, turned.table, turned.rot)
        return t if not unit else t / torch.sqrt(t.pow(2).mean(-1, keepdim=True) + eps)
    x = qkv[..., :heads.packed]
    x = x if bias is None else x.float() + bias.float()
    q = norm(x[..., :heads.q * heads.dk], heads.q, qw)
    if temperature is not None:
        q = q * query_temperature(positions.clamp_min(0), temperature[0], temperature[1])[..., None, None]
    if not heads.own:
        return q.to(qkv.dtype), None, None
    k, v = x[..., heads.q * heads.dk:].split([heads.kv * heads.dk, heads.kv * heads.dv], -1)
    return q.to(qkv.dtype), norm(k, heads.kv, kw).to(qkv.dtype), v.reshape(R, S, heads.kv, heads.dv).to(qkv.dtype)


def _slots(pages: Pages, positions: torch.Tensor) -> torch.Tensor:
    R = positions.shape[0]
    rows = torch.arange(R, device=positions.device) if pages.row_ids is None else pages.row_ids.long()
    p = positions.clamp_min(0).long()
    return pages.table[rows[:, None], p // pages.page_size].long() * pages.page_size + p % pages.page_size


def qk_norm_append(qkv, heads: Heads, qw, kw, eps: float, temperature, positions, pages: Pages, bias=None, turned: Optional[Turned] = None,
                   unit: bool = False) -> torch.Tensor:
    """-> ``[R, S, H + 2 G, D]`` (queries and keys after ``prepare_reference``'s steps, values; every head padded with zeros to the pool's width), with the keys and
    values of the live positions written to the pools; ``[R, S, H, D]`` and nothing written for a layer without its own keys and values.
    ``positions`` int32 ``[R, S]``, below 0 = padding."""
    R, S, _ = qkv.shape
    D = pages.k.shape[-1]
    if L.use_cuda(qkv):
        qkv = qkv.contiguous()
        qw, kw, bias = (None if w is None else w.detach().to(qkv.dtype).contiguous() for w in (qw, kw, bias))
        if per_head(heads, qw, kw) or bias is not None or not heads.own or heads.gated or turned is not None or unit:
            if temperature is not None or not (per_head(heads, qw, kw) or qw is None or heads.q == heads.kv == 1):
                raise NotImplementedError("a projection with a bias, gates, a rotation or queries alone is built for norms per head and without a query "
                                          "temperature")
            if unit and (qw is not None or kw is not None):
                raise NotImplementedError("heads pass one norm: with a weight in front of the rotation, or without one behind it")
            rot, table = (None, None) if turned is None else turned
            G = heads.kv if heads.own else 0
            packed = torch.empty(R, S, heads.q + 2 * G, D, dtype=qkv.dtype, device=qkv.device)
            L.check(L.load().dewb_head_norm_append(L.ptr(qkv), c_ll(qkv.shape[-1]), L.ptr(bias), L.ptr(qw), L.ptr(kw), c_float(eps), c_int(int(unit)),
                                                   L.ptr(table), c_int(0 if rot is None else rot.dims), c_int(int(rot is not None and rot.interleaved)),
                                                   L.ptr(positions), c_int(R), c_int(S), c_int(heads.q), c_int(G), c_int(heads.dk), c_int(heads.dv), c_int(D), L.ptr(packed),
                                                   L.ptr(pages.k), L.ptr(pages.v), L.ptr(pages.table), c_int(pages.page_size), c_int(pages.table.shape[1]),
                                                   L.ptr(pages.row_ids), c_int(int(qkv.dtype == torch.float32)), L.stream_ptr()), "head_norm_append")
            L.count_launches()
            return packed
        packed = torch.empty(R, S, heads.q + 2 * heads.kv, D, dtype=qkv.dtype, device=qkv.device)
        coef, every = temperature if temperature is not None else (0.0, 0)
        L.check(L.load().dewb_qk_norm_append(L.ptr(qkv), L.ptr(qw), L.ptr(kw), c_float(eps), c_float(coef), c_int(every), L.ptr(positions), c_int(R),
                                             c_int(S), c_int(heads.q), c_int(heads.kv), c_int(heads.dk), c_int(heads.dv), c_int(D), L.ptr(packed),
                                             L.ptr(pages.k), L.ptr(pages.v), L.ptr(pages.table), c_int(pages.page_size), c_int(pages.table.shape[1]),
                                             L.ptr(pages.row_ids), c_int(int(qkv.dtype == torch.float32)), L.stream_ptr()), "qk_norm_append")
        L.count_launches()
        return packed
    q, k, v = prepare_reference(qkv, heads, qw, kw, eps, temperature, positions, bias, turned, unit)
    pad = lambda t: torch.nn.functional.pad(t, (0, D - t.shape[-1]))
    if not heads.own:
        return pad(q)
    q, k, v = pad(q), pad(k), pad(v)
    slots, live = _slots(pages, positions), positions >= 0
    for pool, t in ((pages.k, k), (pages.v, v)):
        pool.view(-1, heads.kv, D)[slots[live]] = t[live].to(pool.dtype)
    return torch.cat([q, k, v], 2)


def seen_keys(positions: torch.Tensor, n: int, visible: Visible = PLAIN) -> torch.Tensor:
    """``[R, S, n]``: which of the first ``n`` positions a query at ``positions [R, S]`` sees."""
    j = torch.arange(n, device=positions.device)[None, None]
    seen = j <= positions[..., None]
    if visible.chunk:
        seen = seen & (j >= (positions.clamp_min(0) // visible.chunk * visible.chunk)[..., None])
    if visible.window:
        seen = seen & ((j > positions[..., None] - visible.window) | (j < visible.keep))
    return seen


def softmax_with_sinks(s: torch.Tensor, sinks: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the last axis of ``s [R, H, S, n]`` with each head's sink in the denominator; rows that see nothing give zeros."""
    if sinks is None:
        return torch.nan_to_num(torch.softmax(s, -1))
    sink = sinks.float().view(1, -1, 1, 1).expand(*s.shape[:3], 1)
    return torch.softmax(torch.cat([s, sink], -1), -1)[..., :-1]


def weights_of(s: torch.Tensor, seen: torch.Tensor, visible: Visible) -> torch.Tensor:
    """The keys' weights from their scaled scores ``s [R, H, S, n]`` and ``seen [R, S, n]``."""
    if visible.gain is not None:
        s = s * visible.gain.float().view(1, -1, 1, 1)
    if visible.softcap:
        s = visible.softcap * torch.tanh(s / visible.softcap)
    if visible.sigmoid is not None:
        return torch.sigmoid(s + visible.sigmoid.float().view(1, -1, 1, 1)) * seen[:, None]
    return softmax_with_sinks(s.masked_fill(~seen[:, None], float("-inf")), visible.sinks)


def paged_attend_reference(q, heads: Heads, positions, pages: Pages, scale: float, visible: Visible = PLAIN) -> torch.Tensor:
    R, S = positions.shape
    D = pages.k.shape[-1]
    n = int(positions.max()) + 1
    if n <= 0:
        return q.new_zeros(R, S, heads.q, heads.dv)
    slots = _slots(pages, torch.arange(n, device=q.device)[None].expand(R, n))
    kc = pages.k.view(-1, heads.kv, D)[slots].float().repeat_interleave(heads.q // heads.kv, 2)          # [R, n, H, D]
    vc = pages.v.view(-1, heads.kv, D)[slots][..., :heads.dv].float().repeat_interleave(heads.q // heads.kv, 2)
    seen = seen_keys(positions, n, visible)                                                              # [R, S, n]
    # what the pool holds beyond a row's own tokens is another row's, or nothing: it must not reach the sums
    own = (torch.arange(n, device=q.device)[None] <= positions.amax(1, keepdim=True))[..., None, None]
    kc, vc = torch.where(own, kc, torch.zeros_like(kc)), torch.where(own, vc, torch.zeros_like(vc))
    p = weights_of(torch.einsum("rshd,rnhd->rhsn", q[..., :D].float(), kc) * scale, seen, visible)
    return torch.einsum("rhsn,rnhd->rshd", p, vc).to(q.dtype)


def head_gate_reference(o: torch.Tensor, gate: Optional[torch.Tensor], dv: int) -> torch.Tensor:
    o = o[..., :dv]
    return o if gate is None else (o.float() * torch.sigmoid(gate.float()).unsqueeze(-1)).to(o.dtype)


def head_gate(o: torch.Tensor, gate: Optional[torch.Tensor], dv: int) -> torch.Tensor:
    """``o [..., H, D]`` times the sigmoid of ``gate [..., H]`` (columns of the projection will do), cut to ``dv`` values a head."""
    if gate is None or not L.use_cuda(o):
        return head_gate_reference(o, gate, dv)
    o = o.contiguous()
    H, D = o.shape[-2:]
    tokens = o.numel() // (H * D)
    if gate.stride(-1) != 1 or any(gate.shape[i] > 1 and gate.stride(i) != gate.stride(i + 1) * gate.shape[i + 1] for i in range(gate.dim() - 2)):
        gate = gate.contiguous()
    out = torch.empty(*o.shape[:-1], dv, dtype=o.dtype, device=o.device)
    L.check(L.load().dewb_head_gate(L.ptr(o), L.ptr(gate), c_ll(gate.stride(-2)), L.ptr(out), c_ll(tokens), c_int(H), c_int(dv), c_int(D),
                                    c_int(int(o.dtype == torch.float32)), L.stream_ptr()), "head_gate")
    L.count_launches()
    return out


def paged_attend(q: torch.Tensor, heads: Heads, positions: torch.Tensor, pages: Pages, scale: float, kernel: Optional[str] = None,
                 visible: Visible = PLAIN, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``q [R, S, H, D]`` (a view into the packed tensor will do: unit stride in a head, heads next to each other) -> ``[R, S, H, dv]``, times the
    sigmoid of ``gate [R, S, H]`` where given.  ``kernel`` forces ``mma`` (bf16 pools of 64, 128, 256) or ``general``."""
    if not L.use_cuda(q):
        return head_gate_reference(paged_attend_reference(q, heads, positions, pages, scale, visible), gate, heads.dv)
    R, S, H, D = q.shape
    if q.stride(3) != 1 or q.stride(2) != D or (R > 1 and q.stride(0) != S * q.stride(1)):
        q = q.contiguous()
    out = torch.empty(R, S, H, heads.dv, dtype=q.dtype, device=q.device)
    if gate is not None and (gate.stride(2) != 1 or (R > 1 and gate.stride(0) != S * gate.stride(1))):
        gate = gate.contiguous()
    extras = (c_int(visible.chunk or 0), c_int(visible.window or 0), c_int(visible.keep), c_float(visible.softcap), L.ptr(visible.sinks), L.ptr(gate), c_ll(0 if gate is None else gate.stride(1)),
              L.ptr(visible.gain), L.ptr(visible.sigmoid))
    if (kernel or ("mma" if q.dtype == torch.bfloat16 and D in (64, 128, 256) else "general")) == "mma":
        L.check(L.load().dewb_paged_attend_mma(L.ptr(q), c_ll(q.stride(1)), L.ptr(pages.k), L.ptr(pages.v), L.ptr(positions), c_int(R), c_int(S), c_int(H),
                                               c_int(heads.kv), c_int(heads.dv), c_int(D), c_float(scale), *extras, L.ptr(out), L.ptr(pages.table),
                                               c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids), L.stream_ptr()), "paged_attend_mma")
        L.count_launches()
        return out
    L.check(L.load().dewb_paged_attend(L.ptr(q), c_ll(q.stride(1)), L.ptr(pages.k), L.ptr(pages.v), L.ptr(positions), c_int(R), c_int(S), c_int(H),
                                       c_int(heads.kv), c_int(heads.dk), c_int(heads.dv), c_int(D), c_float(scale), *extras, L.ptr(out), L.ptr(pages.table),
                                       c_int(pages.page_size), c_int(pages.table.shape[1]), L.ptr(pages.row_ids),
                                       c_int(int(q.dtype == torch.float32)), L.stream_ptr()), "paged_attend")
    L.count_launches()
    return out
