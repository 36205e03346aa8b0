"""Linear attention with a constant decay per head over a call's tokens, with the state carried between calls
(``csrc/kernels/decayed_recurrence.cu``): ``S_t = decay S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t``.

Input is the packed projection ``[R, S, H dk | H dk | H dv]``; positions below 0 are padding at the end of a row, and a row whose first
position is 0 starts from a zero state.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch
import torch.nn.functional as F

from . import library as L

c_int = ctypes.c_int


def decayed_attention_reference(qkv, decay, H: int, dk: int, dv: int, state=None, positions=None, row_ids=None, silu: bool = True):
    """Token by token in fp32.  ``state [store rows, H, dk, dv]`` is updated in place when given."""
    R, S, _ = qkv.shape
    x = F.silu(qkv) if silu else qkv
    q, k, v = x.float().split([H * dk, H * dk, H * dv], -1)
    q, k, v = q.view(R, S, H, dk), k.view(R, S, H, dk), v.view(R, S, H, dv)
    a = decay.float().view(1, H, 1, 1)
    pos = positions if positions is not None else torch.arange(S, device=qkv.device)[None].expand(R, S)
    rows = torch.arange(R, device=qkv.device) if row_ids is None else row_ids.long()
    st = torch.zeros(R, H, dk, dv, device=qkv.device)
    if state is not None:
        st = torch.where((pos[:, 0] > 0).view(R, 1, 1, 1), state[rows], st)
    outs = []
    for t in range(S):
        live = (pos[:, t] >= 0).view(R, 1, 1)
        st = torch.where(live.unsqueeze(-1), st * a + torch.einsum("rhk,rhv->rhkv", k[:, t], v[:, t]), st)
        outs.append(torch.where(live, torch.einsum("rhk,rhkv->rhv", q[:, t], st), torch.zeros_like(v[:, t])))
    if state is not None:
        seen = pos[:, 0] >= 0
        state[rows[seen]] = st[seen]
    return torch.stack(outs, 1).to(qkv.dtype)


def chunks_ok(qkv: torch.Tensor, dk: int, dv: int) -> bool:
    return qkv.dtype == torch.bfloat16 and dk % 8 == 0 and dv % 8 == 0 and 8 <= dk <= 128 and qkv.data_ptr() % 16 == 0


def decayed_attention(qkv: torch.Tensor, decay: torch.Tensor, H: int, dk: int, dv: int, state: Optional[torch.Tensor] = None,
                      positions: Optional[torch.Tensor] = None, row_ids: Optional[torch.Tensor] = None, silu: bool = True, kernel: Optional[str] = None) -> torch.Tensor:
    """``qkv [R, S, H (2 dk + dv)] -> [R, S, H, dv]``.  ``positions`` int32 ``[R, S]``, ``row_ids`` int32 (call row -> store row).
    ``kernel`` forces ``chunks`` (tensor cores, bf16) or ``sequence`` (fp32 arithmetic, any widths) for a call of several tokens."""
    R, S, _ = qkv.shape
    if not L.use_cuda(qkv) or qkv.dtype not in (torch.bfloat16, torch.float32):
        return decayed_attention_reference(qkv, decay, H, dk, dv, state, positions, row_ids, silu)
    qkv, decay = qkv.contiguous(), decay.to(qkv.device, torch.float32).contiguous()
    if positions is None:
        positions = torch.arange(S, device=qkv.device, dtype=torch.int32)[None].expand(R, S)
    pos = positions.to(torch.int32).contiguous()
    rows = None if row_ids is None else row_ids.to(torch.int32).contiguous()
    out = torch.empty(R, S, H, dv, dtype=qkv.dtype, device=qkv.device)
    fp32 = c_int(int(qkv.dtype == torch.float32))
    lib = L.load()
    if S == 1 and state is not None:
        L.check(lib.dewb_decayed_step(L.ptr(qkv), L.ptr(decay), L.ptr(state), L.ptr(pos), L.ptr(rows), c_int(R), c_int(H), c_int(dk), c_int(dv),
                                      c_int(int(silu)), L.ptr(out), fp32, L.stream_ptr()), "decayed_step")
    elif (kernel or ("chunks" if chunks_ok(qkv, dk, dv) else "sequence")) == "chunks":
        L.check(lib.dewb_decayed_chunks(L.ptr(qkv), L.ptr(decay), L.ptr(state), L.ptr(pos), L.ptr(rows), c_int(R), c_int(S), c_int(H), c_int(dk),
                                        c_int(dv), c_int(int(silu)), L.ptr(out), L.stream_ptr()), "decayed_chunks")
    else:
        L.check(lib.dewb_decayed_sequence(L.ptr(qkv), L.ptr(decay), L.ptr(state), L.ptr(pos), L.ptr(rows), c_int(R), c_int(S), c_int(H), c_int(dk),
                                          c_int(dv), c_int(int(silu)), L.ptr(out), fp32, L.stream_ptr()), "decayed_sequence")
    L.count_launches()
    return out
