"""Row operations of decoders whose residual is a bundle of fp32 streams (``csrc/kernels/residual_streams.cu``), each with its plain
PyTorch form: the CPU path, the form autograd differentiates, and what the GPU tests compare against.

``stream_step`` is the residual step between two sub-layers in one pass over the streams: the pending write of the sub-layer that just
ran, the read of the next, and its norm.  One stream with unit weights is the ordinary fp32 residual.
"""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional, Tuple

import torch
import torch.nn.functional as F

from . import library as L

c_ll, c_int, c_float = ctypes.c_longlong, ctypes.c_int, ctypes.c_float
MAX_STREAMS = 16


class Write(NamedTuple):
    """A sub-layer's output on its way into the streams: ``H'[t] = sum_s mix[s, t] H[s] + out[t] * (gain * scale * y + gain2 * scale2 * y2)``.  Without
    ``mix`` and ``out`` every stream keeps itself and takes ``y``; with ``weight``, ``y`` passes an RMS norm (``weight``, ``eps``) first; ``y2`` is the second
    of two sub-layers that join together (``gain2`` None: ``gain``)."""
    y: torch.Tensor
    scale: Optional[torch.Tensor] = None
    mix: Optional[torch.Tensor] = None
    out: Optional[torch.Tensor] = None
    weight: Optional[torch.Tensor] = None
    eps: float = 0.0
    y2: Optional[torch.Tensor] = None
    scale2: Optional[torch.Tensor] = None
    gain: float = 1.0
    gain2: Optional[float] = None

    @property
    def second(self) -> float:
        return self.gain if self.gain2 is None else self.gain2


class Join(NamedTuple):
    """What joins one plain stream beside the sub-layers' outputs: ``add [d]``, and ``gain`` times the rows of ``table [vocab, d]`` at ``tokens [...]``."""
    add: Optional[torch.Tensor] = None
    table: Optional[torch.Tensor] = None
    tokens: Optional[torch.Tensor] = None
    gain: float = 1.0


def _kernel_ok(x: torch.Tensor, *others) -> bool:
    """On a GPU the kernels run unless autograd has to see through the operation."""
    if x.dtype not in (torch.bfloat16, torch.float32) or not L.use_cuda(x):
        return False
    return not (torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in (x, *others)))


def _as(t: Optional[torch.Tensor], dtype) -> Optional[torch.Tensor]:
    return None if t is None else t.detach().to(dtype).contiguous()


def layer_norm_reference(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    xf = x.float()
    dev = xf - xf.mean(-1, keepdim=True)
    return dev / torch.sqrt(dev.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def embed_streams(tokens: torch.Tensor, positions: Optional[torch.Tensor], embed: torch.Tensor, pos: Optional[torch.Tensor], n: int,
                  gain: float = 1.0) -> torch.Tensor:
    """``[B, S]`` tokens (and positions, below 0 = padding) -> fp32 streams ``[B, S, n, d]``, all equal to ``gain`` times the embedding plus the learned
    position vector."""
    B, S = tokens.shape
    d = embed.shape[1]
    if pos is not None and positions is None:
        positions = torch.arange(S, device=tokens.device)[None].expand(B, S)
    if _kernel_ok(embed, pos):
        H = torch.empty(B, S, n, d, dtype=torch.float32, device=embed.device)
        tk = tokens.to(torch.int64).contiguous()
        p32 = None if pos is None else positions.to(torch.int32).contiguous()
        e, p = embed.detach().contiguous(), _as(pos, embed.dtype)
        L.check(L.load().dewb_embed_streams(L.ptr(tk), L.ptr(p32), L.ptr(e), L.ptr(p), L.ptr(H), c_ll(B * S), c_int(n), c_int(d), c_int(embed.shape[0]),
                                            c_int(0 if pos is None else pos.shape[0]), c_float(gain), c_int(int(embed.dtype == torch.float32)), L.stream_ptr()), "embed_streams")
        L.count_launches()
        return H
    x = F.embedding(tokens, embed).float() * gain
    if pos is not None:
        x = x + F.embedding(positions.long().clamp_min(0), pos).float()
    return x.unsqueeze(2).expand(B, S, n, d).contiguous()


def stream_step_reference(H, write: Optional[Write], read, weight, eps: float, dtype, norm: str = "layer", around: float = 0.0, join: Optional[Join] = None):
    if write is not None:
        y = write.y.float()
        if write.weight is not None:
            y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + write.eps) * write.weight.float()
        if write.scale is not None:
            y = y * write.scale.float()
        y = y * write.gain
        if write.y2 is not None:
            y = y + write.second * (write.y2.float() if write.scale2 is None else write.y2.float() * write.scale2.float())
        kept = H if write.mix is None else torch.einsum("st,...sd->...td", write.mix.float(), H)
        H = kept + (y.unsqueeze(-2) if write.out is None else write.out.float()[:, None] * y.unsqueeze(-2))
    if join is not None:
        if join.table is not None:
            H = H + join.gain * F.embedding(join.tokens, join.table).float().unsqueeze(-2)
        if join.add is not None:
            H = H + join.add.float()
    if weight is None:
        return None, H
    u = H.sum(-2) if read is None else torch.einsum("s,...sd->...d", read.float(), H)
    weight = weight.float() + around
    if norm == "layer":
        return layer_norm_reference(u, weight, eps).to(dtype), H
    return (u / torch.sqrt(u.pow(2).mean(-1, keepdim=True) + eps) * weight.float()).to(dtype), H


def stream_step(H: torch.Tensor, write: Optional[Write], read: Optional[torch.Tensor], weight: Optional[torch.Tensor], eps: float, dtype,
                norm: str = "layer", around: float = 0.0, join: Optional[Join] = None) -> Tuple[Optional[torch.Tensor], torch.Tensor]:
    """``(norm(sum_s read[s] H'[s]) * (around + weight), H')`` with ``H'`` the streams after ``write`` (None: as they are); ``read`` None: all ones.  ``H [..., n, d]`` fp32;
    on a GPU outside autograd ``H`` is updated in place.  ``weight`` None: the write alone; a ``weight`` of one number counts for all coordinates.  ``join``:
    what else comes in behind the write (one stream)."""
    if norm not in ("layer", "rms"):
        raise ValueError(f"unknown norm {norm!r}; known: layer, rms")
    n, d = H.shape[-2:]
    if join is not None and n != 1:
        raise NotImplementedError("what joins beside the sub-layers is built for one stream")
    tensors = (weight, read) + (() if write is None else (write.y, write.scale, write.mix, write.out, write.weight, write.y2, write.scale2)) + \
        (() if join is None else (join.add, join.table))
    if n > MAX_STREAMS or not H.is_contiguous() or not _kernel_ok(H, *tensors) or dtype not in (torch.bfloat16, torch.float32):
        return stream_step_reference(H, write, read, weight, eps, dtype, norm, around, join)
    rows = H.numel() // (n * d)
    normed = None if weight is None else torch.empty(*H.shape[:-2], d, dtype=dtype, device=H.device)
    y = y_weight = scale = mix = out = y2 = scale2 = None
    if write is not None:
        y, scale, mix, out = _as(write.y, dtype), _as(write.scale, dtype), _as(write.mix, torch.float32), _as(write.out, torch.float32)
        y_weight, y2, scale2 = _as(write.weight, dtype), _as(write.y2, dtype), _as(write.scale2, dtype)
    r, w = _as(read, torch.float32), _as(weight, dtype)
    add, table, tokens = (None, None, None) if join is None else (_as(join.add, dtype), _as(join.table, dtype), join.tokens)
    tokens = None if tokens is None else tokens.to(torch.int64).contiguous()
    L.check(L.load().dewb_stream_step(L.ptr(H), L.ptr(y), L.ptr(y_weight), L.ptr(scale), L.ptr(mix), L.ptr(out), L.ptr(r), L.ptr(w), L.ptr(normed), c_ll(rows),
                                      c_int(n), c_int(d), c_float(0.0 if write is None else write.eps), c_float(eps), c_int(int(norm == "rms")),
                                      L.ptr(y2), L.ptr(scale2), c_float(1.0 if write is None else write.gain), c_float(1.0 if write is None else write.second),
                                      c_float(around), c_int(int(w is not None and w.dim() == 0)), L.ptr(add), L.ptr(table), L.ptr(tokens),
                                      c_int(0 if table is None else table.shape[0]), c_float(1.0 if join is None else join.gain),
                                      c_int(int(dtype == torch.float32)), L.stream_ptr()), "stream_step")
    L.count_launches()
    return normed, H


def clamped_glu_reference(gu: torch.Tensor, limit: float, alpha: float = 1.702) -> torch.Tensor:
    g, u = gu.float().chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + 1.0)).to(gu.dtype)


def clamped_glu(gu: torch.Tensor, limit: float, alpha: float = 1.702) -> torch.Tensor:
    """``[..., 2F]`` (gate half, then linear half) -> ``[..., F]``: ``g sigmoid(alpha g) (u + 1)`` of the clamped halves."""
    if not _kernel_ok(gu):
        return clamped_glu_reference(gu, limit, alpha)
    gu = gu.contiguous()
    Fh = gu.shape[-1] // 2
    out = torch.empty(*gu.shape[:-1], Fh, dtype=gu.dtype, device=gu.device)
    L.check(L.load().dewb_clamped_glu(L.ptr(gu), L.ptr(out), c_ll(gu.numel() // (2 * Fh)), c_int(Fh), c_float(limit), c_float(alpha),
                                      c_int(int(gu.dtype == torch.float32)), L.stream_ptr()), "clamped_glu")
    L.count_launches()
    return out


def gelu_glu_reference(gu: torch.Tensor) -> torch.Tensor:
    g, u = gu.chunk(2, -1)
    return F.gelu(g, approximate="tanh") * u


def gelu_glu(gu: torch.Tensor) -> torch.Tensor:
    """``[..., 2F]`` (gate half, then linear half) -> ``[..., F]``: ``gelu(gate) * up``, the tanh form."""
    if not _kernel_ok(gu):
        return gelu_glu_reference(gu)
    gu = gu.contiguous()
    Fh = gu.shape[-1] // 2
    out = torch.empty(*gu.shape[:-1], Fh, dtype=gu.dtype, device=gu.device)
    L.check(L.load().dewb_gelu_glu(L.ptr(gu), L.ptr(out), c_ll(gu.numel() // (2 * Fh)), c_int(Fh), c_int(int(gu.dtype == torch.float32)), L.stream_ptr()),
            "gelu_glu")
    L.count_launches()
    return out


def softcap_reference(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x.float() / cap)


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap tanh(x / cap)`` in fp32."""
    if not _kernel_ok(x):
        return softcap_reference(x, cap)
    x = x.contiguous()
    n = x.shape[-1]
    out = torch.empty(x.shape, dtype=torch.float32, device=x.device)
    L.check(L.load().dewb_softcap(L.ptr(x), L.ptr(out), c_ll(x.numel() // max(n, 1)), c_int(n), c_float(cap), c_int(int(x.dtype == torch.float32)),
                                  L.stream_ptr()), "softcap")
    L.count_launches()
    return out


def sigmoid_gated_norm_reference(x, gate, w, eps: float) -> torch.Tensor:
    xf = x.float()
    return (xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float() * torch.sigmoid(gate.float())).to(gate.dtype)


def sigmoid_gated_norm(x: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """``RMSnorm(x) * w * sigmoid(gate)`` over the last axis (linear attention's output gate)."""
    if x.dtype != gate.dtype or not _kernel_ok(x, gate, w):
        return sigmoid_gated_norm_reference(x, gate, w, eps)
    x, gate, w = x.contiguous(), gate.contiguous(), _as(w, x.dtype)
    d = x.shape[-1]
    out = torch.empty_like(gate)
    L.check(L.load().dewb_sigmoid_gated_norm(L.ptr(x), L.ptr(gate), L.ptr(w), L.ptr(out), c_ll(x.numel() // d), c_int(d), c_float(eps),
                                             c_int(int(x.dtype == torch.float32)), L.stream_ptr()), "sigmoid_gated_norm")
    L.count_launches()
    return out
