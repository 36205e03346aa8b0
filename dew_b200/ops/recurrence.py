"""Recurrences over a matrix state per head whose decays come from the token (``csrc/kernels/gated_recurrence.cu``, whose head gives the equations, and
``gated_chunks.cu``, the tensor-core form for several tokens in bf16): the gated
delta rule, the matrix memory with exponential gates, and the state with a decay per key channel and a bonus for the token itself.  Each takes a call's
tokens as ``Rows`` and keeps its state between calls; the plain forms go token by token and autograd differentiates them.
"""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional

import torch
import torch.nn.functional as F

from . import library as L
from .token_mix import Rows, kernel_ok, rows_of, same, whole

DELTA, MEMORY, WKV = 0, 1, 2


_FIELDS = (("q k v", ctypes.c_void_p), ("q_stride k_stride v_stride", ctypes.c_longlong),
           ("gates bias0 bias1 log_decay u state n m n_before m_before positions lengths row_ids out", ctypes.c_void_p), ("scale cap", ctypes.c_float),
           ("R S H G dk dv", ctypes.c_int))


class _Args(ctypes.Structure):
    """``dewb_gated_args`` of ``csrc/common/gated_rule.cuh``."""
    _fields_ = [(name, kind) for names, kind in _FIELDS for name in names.split()]


class Memory(NamedTuple):
    """What the matrix memory keeps per store row: the state, the normaliser ``[rows, H, dk]`` and the running maximum ``[rows, H]``."""
    S: torch.Tensor
    n: torch.Tensor
    m: torch.Tensor


def _launch(mode: int, q, k, v, rows: Optional[Rows], H: int, G: int, dk: int, dv: int, state=None, scale: float = 1.0, cap: float = 0.0, gates=None, bias0=None,
            bias1=None, log_decay=None, u=None, memory: Optional[Memory] = None, kernel: Optional[str] = None) -> torch.Tensor:
    R, S = q.shape[:2]
    rows = whole(R, S, q.device) if rows is None else rows
    q, k, v = rows_of(q), rows_of(k), rows_of(v)
    out = torch.empty(R, S, H, dv, dtype=q.dtype, device=q.device)
    # ``kernel`` forces ``chunks`` (tensor cores, bf16) or ``sequence`` (token after token in fp32, any widths)
    before = (None, None) if memory is None or (S == 1 and kernel != "chunks") else (memory.n.clone(), memory.m.clone())      # read by every block of a head while one writes
    f32 = lambda t: None if t is None else t.detach().float().contiguous()
    gates, bias0, bias1, log_decay, u = f32(gates), f32(bias0), f32(bias1), f32(log_decay), same(u, q.dtype)
    at = lambda t: 0 if t is None else t.data_ptr()
    n, m = (None, None) if memory is None else (memory.n, memory.m)
    whole_pieces = q.dtype == torch.bfloat16 and dk <= 128 and not any(n % 8 for n in (dk, dv, q.stride(1), k.stride(1), v.stride(1))) \
        and not any(at(t) % 16 for t in (q, k, v, log_decay))
    chunks = (kernel or ("chunks" if S > 1 and whole_pieces else "sequence")) == "chunks"
    if chunks and not whole_pieces:
        raise ValueError("the chunked form takes bf16 heads of whole 16-byte pieces, keys up to 128 wide")
    args = _Args(at(q), at(k), at(v), q.stride(1), k.stride(1), v.stride(1), at(gates), at(bias0), at(bias1), at(log_decay), at(u), at(state), at(n), at(m),
                 at(before[0]), at(before[1]), at(rows.positions), at(rows.lengths), at(rows.row_ids), at(out), scale, cap, R, S, H, G, dk, dv)
    if chunks:
        L.check(L.load().dewb_gated_chunks(ctypes.c_int(mode), ctypes.byref(args), L.stream_ptr()), "gated_chunks")
    else:
        L.check(L.load().dewb_gated_recurrence(ctypes.c_int(mode), ctypes.byref(args), ctypes.c_int(int(q.dtype == torch.float32)), L.stream_ptr()),
                "gated_recurrence")
    L.count_launches()
    return out


def _tokens(rows: Rows, states, fresh, body, out_shape, dtype):
    """Token by token: ``body(t, states) -> (states, output)``; ``fresh`` are the states of a row that starts, ``states`` the stored ones (or None), updated
    in place."""
    R, S = rows.positions.shape
    at, first = rows.store_rows(), rows.positions[:, 0]
    over = lambda flag, t: flag.view(R, *([1] * (t.dim() - 1)))
    now = [f if s is None else torch.where(over(first > 0, f), s[at], f) for s, f in zip(states, fresh)]
    outs = []
    for t in range(S):
        live = rows.positions[:, t] >= 0
        new, o = body(t, now)
        now = [torch.where(over(live, a), a, b) for a, b in zip(new, now)]
        outs.append(torch.where(over(live, o), o, torch.zeros_like(o)))
    seen = first >= 0
    for s, new in zip(states, now):
        if s is not None:
            s[at[seen]] = new[seen]
    return torch.stack(outs, 1).reshape(out_shape).to(dtype)


def delta_rule_reference(q, k, v, gates, A_log, dt_bias, H: int, G: int, scale: float, rows: Optional[Rows] = None, state=None):
    R, S, _ = q.shape
    rows = whole(R, S, q.device) if rows is None else rows
    dk, dv = q.shape[-1] // G, v.shape[-1] // H
    b, a = gates.float().chunk(2, -1)
    beta, decay = torch.sigmoid(b), torch.exp(-torch.exp(A_log.float()) * F.softplus(a + dt_bias.float(), threshold=60.0))

    def heads(x):
        x = x.float().view(R, S, G, dk)
        return (x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(H // G, 2)
    qf, kf, vf = heads(q) * scale, heads(k), v.float().view(R, S, H, dv)

    def body(t, now):
        st = now[0] * decay[:, t, :, None, None]
        u = beta[:, t, :, None] * (vf[:, t] - torch.einsum("rhkv,rhk->rhv", st, kf[:, t]))
        st = st + kf[:, t].unsqueeze(-1) * u.unsqueeze(-2)
        return [st], torch.einsum("rhkv,rhk->rhv", st, qf[:, t])
    return _tokens(rows, [state], [qf.new_zeros(R, H, dk, dv)], body, (R, S, H, dv), v.dtype)


def delta_rule(q, k, v, gates, A_log, dt_bias, H: int, G: int, scale: Optional[float] = None, rows: Optional[Rows] = None, state=None,
               kernel: Optional[str] = None) -> torch.Tensor:
    """The gated delta rule: ``q, k [R, S, G dk]`` (behind their activation; they are normalised here), ``v [R, S, H dv]``, ``gates [R, S, 2 H]`` fp32 (step
    logits, then decay logits), ``A_log, dt_bias [H]`` -> ``[R, S, H, dv]``; head h uses q and k of head ``h // (H // G)``.  ``state [rows, H, dk, dv]``."""
    dk, dv = q.shape[-1] // G, v.shape[-1] // H
    scale = dk ** -0.5 if scale is None else float(scale)
    if not kernel_ok(q, k, v, gates, A_log, dt_bias):
        return delta_rule_reference(q, k, v, gates, A_log, dt_bias, H, G, scale, rows, state)
    return _launch(DELTA, q, k, v, rows, H, G, dk, dv, state, scale, gates=gates, bias0=A_log, bias1=dt_bias, kernel=kernel)


def matrix_memory_reference(q, k, v, gates, i_bias, f_bias, H: int, cap: float, scale: float, rows: Optional[Rows] = None, memory: Optional[Memory] = None):
    R, S, _ = q.shape
    rows = whole(R, S, q.device) if rows is None else rows
    dk, dv = q.shape[-1] // H, v.shape[-1] // H
    zi, zf = gates.float().chunk(2, -1)
    ins = cap * torch.tanh((zi + i_bias.float()) / cap)
    forgets = F.logsigmoid(cap * torch.tanh((zf + f_bias.float()) / cap))
    qf, kf, vf = q.float().view(R, S, H, dk) * scale, k.float().view(R, S, H, dk), v.float().view(R, S, H, dv)

    def body(t, now):
        st, n, m = now
        top = torch.maximum(forgets[:, t] + m, ins[:, t])
        keep, take = torch.exp(forgets[:, t] + m - top), torch.exp(ins[:, t] - top)
        w = take.unsqueeze(-1) * kf[:, t]
        st = keep[..., None, None] * st + w.unsqueeze(-1) * vf[:, t].unsqueeze(-2)
        n = keep.unsqueeze(-1) * n + w
        den = torch.maximum((n * qf[:, t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        return [st, n, top], torch.einsum("rhkv,rhk->rhv", st, qf[:, t]) / den.unsqueeze(-1)
    fresh = [qf.new_zeros(R, H, dk, dv), qf.new_zeros(R, H, dk), qf.new_zeros(R, H)]
    return _tokens(rows, [None] * 3 if memory is None else list(memory), fresh, body, (R, S, H, dv), v.dtype)


def matrix_memory(q, k, v, gates, i_bias, f_bias, H: int, cap: float, scale: Optional[float] = None, rows: Optional[Rows] = None,
                  memory: Optional[Memory] = None, kernel: Optional[str] = None) -> torch.Tensor:
    """The matrix memory with exponential gates: ``q, k [R, S, H dk]``, ``v [R, S, H dv]``, ``gates [R, S, 2 H]`` fp32 (input logits, then forget logits),
    their biases ``[H]`` -> ``[R, S, H, dv]``."""
    dk, dv = q.shape[-1] // H, v.shape[-1] // H
    scale = dk ** -0.5 if scale is None else float(scale)
    if not kernel_ok(q, k, v, gates, i_bias, f_bias):
        return matrix_memory_reference(q, k, v, gates, i_bias, f_bias, H, cap, scale, rows, memory)
    return _launch(MEMORY, q, k, v, rows, H, H, dk, dv, None if memory is None else memory.S, scale, float(cap), gates, i_bias, f_bias, memory=memory, kernel=kernel)


def bonus_decay_reference(r, k, v, log_decay, u, H: int, rows: Optional[Rows] = None, state=None):
    R, S, _ = r.shape
    rows = whole(R, S, r.device) if rows is None else rows
    dk, dv = r.shape[-1] // H, v.shape[-1] // H
    rf, kf, vf = r.float().view(R, S, H, dk), k.float().view(R, S, H, dk), v.float().view(R, S, H, dv)
    decay = torch.exp(log_decay.float()).view(R, S, H, dk)
    bonus = (rf * u.float() * kf).sum(-1)

    def body(t, now):
        o = torch.einsum("rhkv,rhk->rhv", now[0], rf[:, t]) + bonus[:, t].unsqueeze(-1) * vf[:, t]
        return [decay[:, t].unsqueeze(-1) * now[0] + kf[:, t].unsqueeze(-1) * vf[:, t].unsqueeze(-2)], o
    return _tokens(rows, [state], [rf.new_zeros(R, H, dk, dv)], body, (R, S, H, dv), v.dtype)


def bonus_decay(r, k, v, log_decay, u, H: int, rows: Optional[Rows] = None, state=None, kernel: Optional[str] = None) -> torch.Tensor:
    """The state with a decay per key channel: ``r, k [R, S, H dk]``, ``v [R, S, H dv]``, ``log_decay [R, S, H dk]`` fp32, the bonus ``u [H, dk]`` with which a token
    reads itself -> ``[R, S, H, dv]``."""
    dk, dv = r.shape[-1] // H, v.shape[-1] // H
    if not kernel_ok(r, k, v, log_decay, u):
        return bonus_decay_reference(r, k, v, log_decay, u, H, rows, state)
    return _launch(WKV, r, k, v, rows, H, H, dk, dv, state, log_decay=log_decay, u=u, kernel=kernel)
