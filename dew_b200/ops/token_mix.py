"""What a token takes from its neighbours (short convolutions, token shift) and the small products and norms around a recurrence
(``csrc/kernels/token_mix.cu``), each with its plain PyTorch form: the CPU path and the form autograd differentiates.

A call's rows are described by a ``Rows``: positions below 0 are padding at a row's end, and a row whose first position is 0 starts from nothing.  States are
fp32 tensors over the store's rows, updated in place.
"""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional

import torch
import torch.nn.functional as F

from . import library as L

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float
NARROW_TOKENS = 512          # up to here a narrow product is formed output by output; past it, by a tensor-core product


class Rows(NamedTuple):
    """The rows of one call: ``positions`` int32 ``[R, S]``, ``lengths`` int32 ``[R]`` (the position after a row's last token), ``row_ids`` int32
    (call row -> store row, None: the same)."""
    positions: torch.Tensor
    lengths: torch.Tensor
    row_ids: Optional[torch.Tensor] = None

    def store_rows(self) -> torch.Tensor:
        return torch.arange(self.positions.shape[0], device=self.positions.device) if self.row_ids is None else self.row_ids.long()


def whole(R: int, S: int, device) -> Rows:
    """Rows of ``S`` tokens from their first on."""
    return Rows(torch.arange(S, device=device, dtype=torch.int32)[None].repeat(R, 1), torch.full((R,), S, device=device, dtype=torch.int32))


def kernel_ok(x: torch.Tensor, *others) -> bool:
    """On a GPU the kernels run unless autograd has to see through the operation."""
    if x.dtype not in (torch.bfloat16, torch.float32) or not L.use_cuda(x):
        return False
    return not (torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in (x, *others)))


def rows_of(x: torch.Tensor) -> torch.Tensor:
    """``x [R, S, C]``, or its copy, such that token (r, s) starts at ``(r S + s) stride(1)``."""
    ok = x.stride(-1) == 1 and (x.shape[0] == 1 or x.stride(0) == x.shape[1] * x.stride(1))
    return x if ok else x.contiguous()


def same(t: Optional[torch.Tensor], dtype) -> Optional[torch.Tensor]:
    return None if t is None else t.detach().to(dtype).contiguous()


def conv_tokens_reference(x, w, bias=None, silu: bool = False, rows: Optional[Rows] = None, state: Optional[torch.Tensor] = None):
    R, S, C = x.shape
    taps = w.shape[1]
    rows = whole(R, S, x.device) if rows is None else rows
    u = x.float() if bias is None else x.float() + bias.float()
    before = u.new_zeros(R, taps - 1, C)
    first = rows.positions[:, 0]
    at = rows.store_rows()
    if state is not None and taps > 1:
        before = torch.where((first > 0).view(R, 1, 1), state[at].transpose(1, 2), before)
    u = torch.cat([before, u], 1)
    y = sum(u[:, j:j + S] * w[:, j].float() for j in range(taps))
    if silu:
        y = F.silu(y)
    if state is not None and taps > 1:
        n = (rows.lengths - first).clamp(0, S).long()                             # live tokens of the row; its tail starts there in u
        tail = u.gather(1, (n[:, None] + torch.arange(taps - 1, device=x.device)).unsqueeze(-1).expand(R, taps - 1, C)).transpose(1, 2)
        live = first >= 0
        state[at[live]] = tail[live]
    return torch.where((rows.positions >= 0).unsqueeze(-1), y, torch.zeros_like(y)).to(x.dtype)


def conv_tokens(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, silu: bool = False, rows: Optional[Rows] = None,
                state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x [R, S, C]`` (columns of a wider row will do) through a causal convolution per channel, ``w [C, taps]`` with the token's own weight last, behind
    ``bias [C]``; ``state [store rows, C, taps - 1]`` holds a row's last inputs."""
    if not kernel_ok(x, w, bias):
        return conv_tokens_reference(x, w, bias, silu, rows, state)
    R, S, C = x.shape
    rows = whole(R, S, x.device) if rows is None else rows
    x, wk, b = rows_of(x), same(w, x.dtype), same(bias, x.dtype)
    y = torch.empty(R, S, C, dtype=x.dtype, device=x.device)
    L.check(L.load().dewb_conv_tokens(L.ptr(x), c_ll(x.stride(1)), L.ptr(b), L.ptr(wk), L.ptr(state), L.ptr(rows.positions), L.ptr(rows.lengths),
                                      L.ptr(rows.row_ids), c_int(R), c_int(S), c_int(C), c_int(w.shape[1]), c_int(int(silu)), L.ptr(y),
                                      c_int(int(x.dtype == torch.float32)), L.stream_ptr()), "conv_tokens")
    L.count_launches(1 if S == 1 or state is None else 2)
    return y


def shift_tokens_reference(x, mu, rows: Optional[Rows] = None, state: Optional[torch.Tensor] = None):
    R, S, d = x.shape
    rows = whole(R, S, x.device) if rows is None else rows
    first, at = rows.positions[:, 0], rows.store_rows()
    before = x.new_zeros(R, 1, d, dtype=torch.float32)
    if state is not None:
        before = torch.where((first > 0).view(R, 1, 1), state[at].unsqueeze(1), before)
    xf = x.float()
    prev = torch.cat([before, xf[:, :-1]], 1)
    out = xf + (prev - xf) * mu.float().view(-1, 1, 1, d)
    if state is not None:
        live = first >= 0
        last = (rows.lengths - first).clamp(1, S).long() - 1
        state[at[live]] = xf[torch.arange(R, device=x.device), last][live]
    return torch.where((rows.positions >= 0).unsqueeze(-1), out, torch.zeros_like(out)).to(x.dtype)


def shift_tokens(x: torch.Tensor, mu: torch.Tensor, rows: Optional[Rows] = None, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``[n, R, S, d]``: the mixes ``x + (x' - x) mu_j`` of every token of ``x [R, S, d]`` with the one before it, for ``mu [n, d]``; ``state [store rows, d]``
    holds a row's last token."""
    if not kernel_ok(x, mu):
        return shift_tokens_reference(x, mu, rows, state)
    R, S, d = x.shape
    rows = whole(R, S, x.device) if rows is None else rows
    x, m = x.contiguous(), same(mu, x.dtype)
    out = torch.empty(m.shape[0], R, S, d, dtype=x.dtype, device=x.device)
    L.check(L.load().dewb_shift_tokens(L.ptr(x), L.ptr(m), L.ptr(state), L.ptr(rows.positions), L.ptr(rows.lengths), L.ptr(rows.row_ids), c_int(R), c_int(S),
                                       c_int(d), c_int(m.shape[0]), L.ptr(out), c_int(int(x.dtype == torch.float32)), L.stream_ptr()), "shift_tokens")
    L.count_launches(1 if S == 1 or state is None else 2)
    return out


def narrow_product(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x [..., d] w [n, d]^T`` in fp32: products whose few outputs must not be rounded (gates, bottlenecks)."""
    if not kernel_ok(x, w):
        return F.linear(x.float(), w.float())
    d, n = x.shape[-1], w.shape[0]
    x2 = x.reshape(-1, d).contiguous()
    wk, T = same(w, x.dtype), x2.shape[0]
    if T > NARROW_TOKENS and x.dtype == torch.bfloat16 and d % 8 == 0:
        from .functional import gemm
        out = torch.empty(T, (n + 7) // 8 * 8, dtype=torch.float32, device=x.device)[:, :n]
        gemm(x2, wk, out=out, kernel="sm100_tcgen05")
        return out.contiguous().view(*x.shape[:-1], n)
    out = torch.empty(T, n, dtype=torch.float32, device=x.device)
    for t0 in range(0, T, 1 << 17):
        t1 = min(T, t0 + (1 << 17))
        L.check(L.load().dewb_narrow_product(L.ptr(x2[t0:t1]), L.ptr(wk), L.ptr(out[t0:t1]), c_ll(t1 - t0), c_int(n), c_int(d),
                                             c_int(int(x.dtype == torch.float32)), L.stream_ptr()), "narrow_product")
        L.count_launches()
    return out.view(*x.shape[:-1], n)


def own_products(x: torch.Tensor, w: torch.Tensor):
    """The products of n inputs ``x [n, R, S, d]`` with weights of their own ``w [n, m, d]``: n tensors ``[R, S, m]``."""
    n, R, S, d = x.shape
    if R * S > 128 or not kernel_ok(x, w):
        from .functional import linear
        return tuple(linear(x[i], w[i]) for i in range(n))
    return torch.bmm(x.view(n, R * S, d), w.to(x.dtype).transpose(1, 2)).view(n, R, S, -1).unbind(0)      # a decode step: one launch


def low_rank_decay(z: torch.Tensor, w2: torch.Tensor, w0: torch.Tensor) -> torch.Tensor:
    """``-exp(w2 tanh(z) + w0)`` in fp32 (the logarithm of a decay per channel): ``z [..., rank]`` fp32, ``w2 [C, rank]``, ``w0 [C]``."""
    if not kernel_ok(z, w2, w0):
        return -torch.exp(F.linear(torch.tanh(z.float()), w2.float(), w0.float()))
    C, rank = w2.shape
    z2 = z.reshape(-1, rank).contiguous()
    wk, bk = w2.detach().contiguous(), same(w0, w2.dtype)
    out = torch.empty(*z.shape[:-1], C, dtype=torch.float32, device=z.device)
    L.check(L.load().dewb_low_rank_decay(L.ptr(z2), c_ll(rank), L.ptr(wk), L.ptr(bk), L.ptr(out), c_ll(z2.shape[0]), c_int(C), c_int(rank),
                                         c_int(int(w2.dtype == torch.float32)), L.stream_ptr()), "low_rank_decay")
    L.count_launches()
    return out


ACTS = {"sigmoid": 0, "silu": 1}


def head_gated_norm_reference(x, gate, w, eps: float, act: str = "silu"):
    xf, z = x.float(), gate.float().reshape(x.shape)
    y = xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * (w.float() if w.numel() == x.shape[-1] else w.float().view(x.shape[-2:]))
    return (y * (F.silu(z) if act == "silu" else torch.sigmoid(z))).to(gate.dtype).flatten(-2)


def head_gated_norm(x: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float, act: str = "silu") -> torch.Tensor:
    """Every head of ``x [R, S, H, d]`` over its root mean square, times ``w`` (``[d]``: one for all heads, or ``[H d]``), times ``act`` of ``gate [R, S, H d]``
    (columns of a wider row will do) -> ``[R, S, H d]``."""
    if act not in ACTS:
        raise ValueError(f"unknown gate activation {act!r}; known: {sorted(ACTS)}")
    R, S, H, d = x.shape
    if x.dtype != gate.dtype or not kernel_ok(x, gate, w):
        return head_gated_norm_reference(x, gate, w, eps, act)
    x, gate, wk = x.contiguous(), rows_of(gate), same(w, x.dtype)
    out = torch.empty(R, S, H * d, dtype=x.dtype, device=x.device)
    L.check(L.load().dewb_head_gated_norm(L.ptr(x), L.ptr(gate), c_ll(gate.stride(1)), L.ptr(wk), c_int(int(wk.numel() == d and H > 1)), c_float(eps),
                                          c_int(ACTS[act]), c_ll(R * S), c_int(H), c_int(d), L.ptr(out), c_int(int(x.dtype == torch.float32)), L.stream_ptr()),
            "head_gated_norm")
    L.count_launches()
    return out
