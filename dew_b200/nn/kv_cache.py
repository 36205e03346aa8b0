"""KV cache: dense or paged pools, optional int8 / fp8-e4m3 storage, decode attention over the pages.

Parity: src/dew/nn/kv_cache.py (``KVCache`` spec :362-408 - ``quantized``, ``page_size``, ``pages``, ``groups``,
``offloaded``; ``quantize`` / ``dequantize`` :411-446 per-token-per-head absmax scales; ``hadamard`` :465-479;
``KVStore.write / attend / decode`` :787-1180; pool layout :1297-1320; ``gather_cache_rows`` :1686).
A decoder whose layers differ in what they keep (heads of other widths, latent rows, recurrent states, a layer that runs several times) gives the
store one ``CacheSlot`` per layer run; ``attend_slot``, ``attend_latent`` and ``state`` then take the place of ``attend``.
Pool layout here: ``[layers, pages, page_size, kv_heads, head_dim]`` for keys and for values, a page table
``[rows, max_pages]`` and ``lengths [rows]``; a dense cache is the special case of one page per row.
"""
from __future__ import annotations

import ctypes
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .. import ops
from ..ops import latent as M
from ..ops import library as L
from ..ops import paged as P
from ..ops import rotary, token_mix

LIMITS = {"int8": 127.0, "float8_e4m3fn": 448.0}
KINDS = {None: 0, "int8": 1, "float8_e4m3fn": 2}


@dataclass(frozen=True)
class KVCache:
    quantized: Optional[str] = None           # None | "int8" | "float8_e4m3fn"
    page_size: Optional[int] = None           # None: dense ("whole") rows
    pages: Optional[int] = None               # pool size; default rows * pages_per_row
    groups: int = 1
    offloaded: bool = False

    def __post_init__(self):
        if self.quantized not in KINDS:
            raise ValueError(f"quantized must be one of {list(KINDS)}, got {self.quantized!r}")


@dataclass(frozen=True)
class CacheSlot:
    """What one run of a layer keeps per row: keys and values of its own head count and widths (with ``latent``, rows of which the first ``value_dim``
    columns are the values too), a recurrent state (a shape, fp32), or nothing: it reads the keys and values of the earlier slot ``source``.  ``more`` names
    further fp32 tensors of a row (the inputs a convolution still needs, a normaliser); ``beside`` is what a second mixer of the same layer keeps, in a slot
    of its own behind those of the layers (``KVStore.beside``)."""
    kv_heads: int = 0
    head_dim: int = 0
    value_dim: int = 0
    state: Optional[Tuple[int, ...]] = None
    source: Optional[int] = None
    latent: bool = False
    more: Tuple[Tuple[str, Tuple[int, ...]], ...] = ()
    beside: Optional["CacheSlot"] = None

    @property
    def stateful(self) -> bool:
        """Whether a row keeps something here that no page holds."""
        return self.state is not None or bool(self.more)


@dataclass
class Call:
    """The integers of one forward call, and its angles, computed once for all its layers.  ``key`` holds the positions tensor itself, so its memory cannot
    be handed to another tensor while this entry can still be found."""
    key: torch.Tensor
    version: int
    capturing: bool
    row_key: Optional[torch.Tensor]
    positions: torch.Tensor                  # int32 [R, S], below 0 = padding
    lengths: torch.Tensor                    # int32 [R]: tokens a row holds after this call's last position (decode: position + 1)
    row_ids: Optional[torch.Tensor]          # int32 store row of each call row, None: the same
    table: torch.Tensor                      # int32 [R, max_pages]: the call rows' page tables
    fresh: Optional[bool] = None             # every row starts at its first token (None: not looked at)
    kept: Dict[int, torch.Tensor] = field(default_factory=dict)      # slot -> this call's packed heads, while later layers read its keys and values
    angles: Dict[rotary.Rotary, torch.Tensor] = field(default_factory=dict)

    @property
    def rows(self) -> token_mix.Rows:
        return token_mix.Rows(self.positions, self.lengths, self.row_ids)

    def turned(self, rot: Optional[rotary.Rotary]) -> Optional[P.Turned]:
        if rot is None:
            return None
        if rot not in self.angles:
            self.angles[rot] = rotary.angles(self.positions, rot)
        return P.Turned(rot, self.angles[rot])


def pool_width(slot: CacheSlot, dtype) -> int:
    """Width of a slot's pool heads: what the bf16 kernels are built for (64, 128, 256) where the head fits, else the head rounded up to 8; latent rows
    are rounded up to 16, and 8 more (the kernel's bank spacing)."""
    if slot.latent:
        return (slot.head_dim + 15) // 16 * 16 + 8
    w = max(slot.head_dim, slot.value_dim)
    if dtype == torch.bfloat16:
        for d in (64, 128, 256):
            if w <= d:
                return d
    return (w + 7) // 8 * 8


def hadamard(x: torch.Tensor) -> torch.Tensor:
    """Fast Walsh-Hadamard transform over the last axis (a power of two), orthonormal; spreads outliers before int8."""
    n = x.shape[-1]
    assert n & (n - 1) == 0
    y = x.float().reshape(-1, n)
    h = 1
    while h < n:
        y = y.view(-1, n // (2 * h), 2, h)
        y = torch.stack([y[:, :, 0] + y[:, :, 1], y[:, :, 0] - y[:, :, 1]], 2).reshape(-1, n)
        h *= 2
    return (y / math.sqrt(n)).reshape(x.shape)


def quantize(x: torch.Tensor, kind: str) -> Tuple[torch.Tensor, torch.Tensor]:
    """Per-token-per-head: ``scale = absmax / limit``; returns (stored values, fp32 scales ``[..., heads]``)."""
    limit = LIMITS[kind]
    amax = x.float().abs().amax(-1)
    scale = torch.where(amax > 0, amax / limit, torch.ones_like(amax))
    y = x.float() / scale[..., None]
    if kind == "int8":
        return y.round().clamp(-127, 127).to(torch.int8), scale
    return y.to(torch.float8_e4m3fn), scale


def dequantize(q: torch.Tensor, scale: torch.Tensor, dtype=torch.float32) -> torch.Tensor:
    return (q.float() * scale[..., None]).to(dtype)


def default_page_table(rows: int, pages_per_row: int, device=None) -> torch.Tensor:
    return torch.arange(rows * pages_per_row, dtype=torch.int32, device=device).reshape(rows, pages_per_row)


class KVStore:
    def __init__(self, spec: KVCache, layers: int, rows: int, max_len: int, kv_heads: int, head_dim: int,
                 dtype=torch.bfloat16, device="cpu", slots: Optional[Sequence[CacheSlot]] = None):
        self.spec = spec
        self.slots = None if slots is None else list(slots)
        self.layer_runs = 0 if slots is None else len(self.slots)
        self.beside: Dict[int, int] = {}             # slot of a layer run -> slot of the second mixer's share of it
        for i in range(self.layer_runs):
            if self.slots[i].beside is not None:
                self.beside[i] = len(self.slots)
                self.slots.append(self.slots[i].beside)
        self.layers, self.rows, self.max_len, self.kv_heads, self.head_dim = layers, rows, max_len, kv_heads, head_dim
        self.page_size = spec.page_size or max_len
        self.max_pages = (max_len + self.page_size - 1) // self.page_size
        self.pages = spec.pages or rows * self.max_pages
        self.kind = KINDS[spec.quantized]
        store = {0: dtype, 1: torch.int8, 2: torch.float8_e4m3fn}[self.kind]
        # one page beyond the addressable pool: writes of padding positions land there, so that a write needs no data-dependent
        # shapes (and therefore no host synchronisation); no page table entry ever names it
        self.states: List[Optional[torch.Tensor]] = []
        self.more: List[Dict[str, torch.Tensor]] = []
        self._call: Optional[Call] = None
        if self.slots is not None:
            if self.kind:
                raise NotImplementedError("quantised storage is built for caches whose layers all keep the same heads")
            for i, s in enumerate(self.slots):
                if s.source is not None and not (0 <= s.source < i and self.slots[s.source].source is None and self.slots[s.source].state is None):
                    raise ValueError(f"slot {i} reads the keys and values of slot {s.source}, which keeps none of its own before it")
            pool = lambda s: None if s.state is not None or s.source is not None else \
                torch.zeros(self.pages + 1, self.page_size, s.kv_heads, pool_width(s, dtype), dtype=dtype, device=device)
            self.k = [pool(s) for s in self.slots]
            self.v = [k if s.latent else pool(s) for k, s in zip(self.k, self.slots)]
            for pools in (self.k, self.v):
                for i, s in enumerate(self.slots):
                    if s.source is not None:
                        pools[i] = pools[s.source]
            self.last_reader = {s.source: i for i, s in enumerate(self.slots) if s.source is not None}
            self.states = [None if s.state is None else torch.zeros(rows, *s.state, dtype=torch.float32, device=device) for s in self.slots]
            self.more = [{n: torch.zeros(rows, *shape, dtype=torch.float32, device=device) for n, shape in s.more} for s in self.slots]
            self.k_scale = self.v_scale = None
        else:
            shape = (layers, self.pages + 1, self.page_size, kv_heads, head_dim)
            self.k = torch.zeros(shape, dtype=store, device=device)
            self.v = torch.zeros(shape, dtype=store, device=device)
            self.k_scale = torch.ones(shape[:-1], dtype=torch.float32, device=device) if self.kind else None
            self.v_scale = torch.ones(shape[:-1], dtype=torch.float32, device=device) if self.kind else None
        self.page_table = default_page_table(rows, self.max_pages, device) if spec.pages is None else \
            torch.zeros(rows, self.max_pages, dtype=torch.int32, device=device)
        self.lengths = torch.zeros(rows, dtype=torch.int32, device=device)
        self.dtype, self.device = dtype, torch.device(device)
        self.row_ids: Optional[torch.Tensor] = None      # rows of the store addressed by the batch rows of a call
        self._scratch = None
        self.chunk_span: Optional[Tuple[int, int]] = None      # (first position, one past the last) of the prefill chunk in flight, when the caller knows
        self.together = True         # whether every row of that chunk starts at its first position

    # ------------------------------------------------------------------ layers that differ (CacheSlot)
    @property
    def keeps_state(self) -> bool:
        """Whether some layer keeps a state (which no page holds: a prompt's prefix cannot be taken from another row's pages)."""
        return any(s.stateful for s in self.slots or ())

    def kept_states(self) -> List[torch.Tensor]:
        """Every tensor of the store that a step moves on instead of adding to."""
        return [t for t in self.states if t is not None] + [t for named in self.more for t in named.values()]

    def call(self, positions: torch.Tensor) -> Call:
        """The integers of the call whose layers pass ``positions [R, S]``: made by the first layer, found by the others."""
        capturing = positions.is_cuda and torch.cuda.is_current_stream_capturing()
        c = self._call
        if c is not None and c.key is positions and c.version == positions._version and c.capturing == capturing and c.row_key is self.row_ids:
            return c
        pos = positions.to(torch.int32).contiguous()
        ids = self.row_ids
        if ids is None and positions.shape[0] > self.rows:
            raise ValueError(f"{positions.shape[0]} rows do not fit a cache of {self.rows}")
        table = self.page_table[: positions.shape[0]] if ids is None else self.page_table[ids]
        self._call = Call(positions, positions._version, capturing, ids, pos, (pos.amax(1) + 1).to(torch.int32),
                          None if ids is None else ids.to(torch.int32), table)
        return self._call

    def is_fresh(self, c: Call) -> bool:
        if self.chunk_span is not None:
            return self.chunk_span[0] == 0
        if c.fresh is None:
            c.fresh = bool((c.positions[:, 0] <= 0).all())
        return c.fresh

    def attend_slot(self, slot: int, qkv: torch.Tensor, heads: P.Heads, positions: torch.Tensor, *, scale: float, eps: float = 1e-6, q_weight=None,
                    k_weight=None, temperature=None, bias=None, chunk: Optional[int] = None, sinks: Optional[torch.Tensor] = None,
                    window: Optional[int] = None, keep: int = 0, softcap: float = 0.0, rot: Optional[rotary.Rotary] = None, unit: bool = False,
                    gain: Optional[torch.Tensor] = None, sigmoid: Optional[torch.Tensor] = None) -> torch.Tensor:
        """A layer's attention from its packed projection ``qkv [R, S, heads.row]``: bias, norms, rotation, temperature, append, causal attention
        against everything the rows hold (or what ``paged.Visible`` leaves of it, times the heads' gates).  -> ``[R, S, H, dv]``.  A
        prompt from its first token takes the tcgen05 flash kernel, a decode step the paged decode kernels, anything else (and fp32) the
        general paged kernel.  A slot with a source appends nothing and reads the source's keys and values."""
        c = self.call(positions)
        source = self.slots[slot].source
        if (source is None) != heads.own:
            raise ValueError(f"slot {slot}: the layer and the cache disagree on whether it has keys and values of its own")
        pages = P.Pages(self.k[slot], self.v[slot], self.page_table, self.page_size, c.row_ids)
        packed = P.qk_norm_append(qkv, heads, q_weight, k_weight, eps, temperature, c.positions, pages, bias, c.turned(rot), unit)
        gate = qkv[..., heads.packed:] if heads.gated else None
        fp32 = lambda name, t: None if t is None else self._fp32_of(slot, name, t)
        visible = P.Visible(chunk, fp32("sinks", sinks), window, keep if window else 0, softcap, fp32("gain", gain), fp32("sigmoid", sigmoid))
        R, S = positions.shape
        H, G = heads.q, heads.kv
        D = packed.shape[-1]
        q = packed[:, :, :H]
        if L.use_cuda(qkv) and qkv.dtype == torch.bfloat16:
            if S == 1 and D in (64, 128, 256):
                return P.head_gate(self._decode_slot(slot, packed, heads, c, scale, visible)[:, None], gate, heads.dv)
            if D in (64, 128) and S % 128 == 0 and self.is_fresh(c):
                from ..ops.flash import Variants, flash_fwd
                if slot in self.last_reader:
                    c.kept[slot] = packed[:, :, H:]
                kv = packed[:, :, H:] if source is None else c.kept.get(source)
                if source is not None and self.last_reader[source] == slot:
                    c.kept.pop(source, None)
                if kv is not None:
                    out, _ = flash_fwd(q, kv[:, :, :G], kv[:, :, G:], True, scale, need_lse=False, var=Variants(visible.window, softcap, visible.sinks, chunk=chunk,
                                                                                                                keep=visible.keep, gain=visible.gain,
                                                                                                                sigmoid=visible.sigmoid))
                    return P.head_gate(out, gate, heads.dv)
        return P.paged_attend(q, heads, c.positions, pages, scale, visible=visible, gate=gate)

    def _fp32_of(self, slot: int, name: str, t: torch.Tensor) -> torch.Tensor:
        """A layer's numbers per head (sinks, factors, biases) as the kernels take them, converted once (again when the parameter changes)."""
        bank = self.__dict__.setdefault("_per_head", {})
        key = (t.data_ptr(), t._version)
        if (slot, name) not in bank or bank[slot, name][0] != key:
            bank[slot, name] = (key, t.detach().float().contiguous())
        return bank[slot, name][1]

    def _decode_slot(self, slot: int, packed: torch.Tensor, heads: P.Heads, c: Call, scale: float, visible: P.Visible = P.PLAIN) -> torch.Tensor:
        lib = L.load()
        R, D, H, G = packed.shape[0], packed.shape[-1], heads.q, heads.kv
        out = torch.empty(R, H, D, dtype=packed.dtype, device=packed.device)
        factors = visible.gain is not None or visible.sigmoid is not None
        if D == 128 and self.page_size % 64 == 0 and H // G <= 8 and hasattr(lib, "dewb_paged_decode_persist") and (R <= 1024 or not factors):
            self._fused_decode(lib, slot, packed, packed.shape[2] * D, c.lengths, R, H, D, visible.window, visible.sinks, out, scale=scale, kv_heads=G, table=c.table,
                               visible=visible)
            return out
        q = packed[:, 0, :H].contiguous()
        share = next(s for s in range(1, H // G + 1) if (H // G) % s == 0 and H // G // s <= 8)     # CTAs that share a key / value head
        splits, longest = 1, min(self.max_len, visible.chunk or self.max_len, visible.window + visible.keep if visible.window else self.max_len)
        while splits < 16 and R * G * share * splits < 592 and longest // (splits * 2) >= 256:
            splits *= 2
        pm, pl, pa = self._partials(R * H * splits, D, q.device)
        L.check(lib.dewb_paged_decode(L.ptr(q), L.ptr(self.k[slot]), L.ptr(self.v[slot]), L.ptr(None), L.ptr(None), L.ptr(c.table), L.ptr(c.lengths),
                                      L.ptr(visible.sinks), L.ptr(out), L.ptr(None), L.ptr(pm), L.ptr(pl), L.ptr(pa), ctypes.c_int(R), ctypes.c_int(H),
                                      ctypes.c_int(G), ctypes.c_int(share), ctypes.c_int(D), ctypes.c_int(self.page_size), ctypes.c_int(self.max_pages),
                                      ctypes.c_int(splits), ctypes.c_float(scale), ctypes.c_int(visible.window or 0), ctypes.c_int(visible.keep),
                                      ctypes.c_int(visible.chunk or 0), ctypes.c_float(visible.softcap), L.ptr(visible.gain), L.ptr(visible.sigmoid), ctypes.c_int(0),
                                      L.stream_ptr()), "paged_decode")
        L.count_launches(2)
        return out

    def _partials(self, n: int, D: int, device):
        """Scratch for ``n`` partial sums of ``D`` values.  The buffers grow apart and never shrink, so that layers of different shapes settle on one
        set (a captured step keeps using what its warm-up left)."""
        have = [0, 0, 0] if self._scratch is None else [t.numel() for t in self._scratch]
        if any(h < w for h, w in zip(have, (n, n, n * D))):
            self._scratch = tuple(t if t is not None and t.numel() >= w else torch.empty(w, dtype=torch.float32, device=device)
                                  for t, w in zip(self._scratch or (None,) * 3, (n, n, n * D)))
        return self._scratch

    def attend_latent(self, slot: int, z: torch.Tensor, queries, up: torch.Tensor, lat: M.Latent, positions: torch.Tensor, *, scale: float, eps: float,
                      q_weight=None, kv_weight=None, gated: bool = False) -> torch.Tensor:
        """A latent attention layer from its input projection ``z [R, S, q_rank | rank | rot_dim (| gate)]``: norms, rotation, append, causal attention
        against everything the rows hold, up-projection, gate.  ``queries`` makes ``[R, S, H * width]`` of the normed query latent; ``up`` is the
        keys' and values' up-projection ``[H * (dim + vdim), rank]``.  -> ``[R, S, H * vdim]``.  Portions whose rows start together form their keys
        in full width and take the tcgen05 flash kernel; decode steps, mixed positions and fp32 stay in the latents' space."""
        c = self.call(positions)
        pages = P.Pages(self.k[slot], self.v[slot], self.page_table, self.page_size, c.row_ids)
        table = c.turned(lat.rotary).table
        cq, made = M.rows(z, lat, q_weight, kv_weight, eps, table, c.positions, pages)
        R, S = positions.shape
        q = queries(cq).view(R, S, lat.heads, lat.width)
        gate = z[..., lat.q_rank + lat.row:] if gated else None
        if L.use_cuda(z) and S > 1 and M.flash_ok(q, lat):
            start = 0 if self.is_fresh(c) else self.chunk_span[0] if self.chunk_span is not None and self.together else None
            if start is not None:
                if start > 0:
                    made = M.gather(lat, c.lengths, start + S, pages)
                return M.flash(M.rotate(q, lat, table), made, up, lat, scale, gate)
        o = M.attend(M.absorb(q, up, lat, table, self.k[slot].shape[-1]), lat, c.positions, pages, scale, self.max_len,
                     lambda n, width: self._partials(n, width, z.device))
        return M.expand(o, up, lat, gate)

    # ------------------------------------------------------------------ latent rows (multi-head latent attention)
    def latent(self, layer: int, width: int) -> torch.Tensor:
        """``[rows, max_len, width]`` per layer: what multi-head latent attention caches per token (its normalised KV latent
        and the shared rotary key) instead of per-head keys and values.  Allocated on first use."""
        bank = self.__dict__.setdefault("_latent", {})
        if layer not in bank:
            bank[layer] = torch.zeros(self.rows, self.max_len, width, dtype=self.dtype, device=self.device)
        return bank[layer]

    def write_latent(self, layer: int, values: torch.Tensor, positions: torch.Tensor) -> None:
        """``values [R, S, width]`` at ``positions [R, S]`` of the selected rows (negative positions are skipped)."""
        R, S = positions.shape
        buf = self.latent(layer, values.shape[-1])
        rows = self._rows(R)[:, None].expand(R, S)
        live = positions >= 0
        buf[rows[live], positions[live].long()] = values[live].to(buf.dtype)

    def read_latent(self, layer: int, width: int, length: int) -> torch.Tensor:
        """The selected rows' first ``length`` cached latents ``[R, length, width]``."""
        buf = self.latent(layer, width)
        rows = self._rows(self.rows if self.row_ids is None else self.row_ids.numel())
        return buf[rows, :length]

    # ------------------------------------------------------------------ addressing
    def select(self, row_ids: Optional[torch.Tensor]) -> "KVStore":
        """Batch row ``i`` of the next calls addresses store row ``row_ids[i]`` (None: identity)."""
        self.row_ids = None if row_ids is None else row_ids.to(self.device, torch.int64)
        return self

    def _rows(self, n: int) -> torch.Tensor:
        return torch.arange(n, device=self.device) if self.row_ids is None else self.row_ids

    def _slots(self, rows: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """Flat pool token index (page * page_size + offset) for (row, position) pairs."""
        page = self.page_table[rows, (positions // self.page_size).long()].long()
        return page * self.page_size + (positions % self.page_size).long()

    # ------------------------------------------------------------------ writes
    def write(self, layer: int, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor) -> None:
        """Store ``k, v [R, S, Hkv, D]`` at ``positions [R, S]`` (negative positions are skipped)."""
        R, S = positions.shape
        rows = self._rows(R)[:, None].expand(R, S).reshape(-1)
        flat = positions.reshape(-1)
        live = flat >= 0
        slots = torch.where(live, self._slots(rows, flat.clamp_min(0)), self.pages * self.page_size)      # padding -> the spare page
        kk, vv = k.reshape(R * S, self.kv_heads, self.head_dim), v.reshape(R * S, self.kv_heads, self.head_dim)
        kp, vp = self.k[layer].reshape(-1, self.kv_heads, self.head_dim), self.v[layer].reshape(-1, self.kv_heads, self.head_dim)
        if self.kind:
            kq, ks = quantize(kk, self.spec.quantized)
            vq, vs = quantize(vv, self.spec.quantized)
            kp[slots], vp[slots] = kq, vq
            self.k_scale[layer].reshape(-1, self.kv_heads)[slots] = ks
            self.v_scale[layer].reshape(-1, self.kv_heads)[slots] = vs
        else:
            kp[slots], vp[slots] = kk.to(kp.dtype), vv.to(vp.dtype)

    def append(self, layer: int, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor) -> None:
        """One token per row: ``k, v [R, Hkv, D]`` written at ``positions [R]``."""
        if L.use_cuda(k) and k.dtype == torch.bfloat16 and self.row_ids is None and k.shape[0] == self.rows:
            lib = L.load()
            # every temporary stays referenced until the launch is enqueued: a temporary released between two `L.ptr` calls hands
            # its block back to the allocator, and the next temporary of the same size would take (and overwrite) it
            kc, vc, pos32 = k.contiguous(), v.contiguous(), positions.to(torch.int32).contiguous()
            L.check(lib.dewb_kv_append(L.ptr(kc), L.ptr(vc), L.ptr(self.k[layer]), L.ptr(self.v[layer]),
                                       L.ptr(self.k_scale[layer] if self.kind else None),
                                       L.ptr(self.v_scale[layer] if self.kind else None), L.ptr(self.page_table),
                                       L.ptr(pos32), ctypes.c_int(k.shape[0]),
                                       ctypes.c_int(self.kv_heads), ctypes.c_int(self.head_dim), ctypes.c_int(self.page_size),
                                       ctypes.c_int(self.max_pages), ctypes.c_int(self.kind), L.stream_ptr()), "kv_append")
            L.count_launches()
            return
        self.write(layer, k[:, None], v[:, None], positions[:, None])

    # ------------------------------------------------------------------ the fused decode step
    def _step_ints(self, positions: torch.Tensor):
        """(positions, lengths) of a decode step as int32, computed once per step: every layer of a forward passes the same
        positions tensor, so the conversions and the ``where`` run for the first layer only."""
        key = (positions.data_ptr(), positions._version, tuple(positions.shape), torch.cuda.is_current_stream_capturing() if positions.is_cuda else False)
        cached = getattr(self, "_ints", None)
        if cached is not None and cached[0] == key:
            return cached[1], cached[2]
        pos32 = positions.to(torch.int32).contiguous()
        lens32 = torch.where(pos32 >= 0, pos32 + 1, torch.zeros_like(pos32))
        self._ints = (key, pos32, lens32)
        return pos32, lens32

    def can_decode_packed(self, qkv: torch.Tensor, Hq: int, softcap: float = 0.0) -> bool:
        return (qkv.is_cuda and qkv.dtype == torch.bfloat16 and qkv.is_contiguous() and self.kind == 0 and self.row_ids is None
                and qkv.shape[0] == self.rows and self.head_dim == 128 and self.page_size % 64 == 0 and not softcap
                and Hq // self.kv_heads <= 8 and os.environ.get("DEWB_DECODE", "stream") == "stream"
                and hasattr(L.load(), "dewb_rope_append"))

    MIN_TILES = 4            # fewest 64-key tiles one CTA of the balanced decode kernel takes (bounds the parts a row is cut into)

    def _fused_decode(self, lib, layer: int, q, q_row_stride: int, lens32, R: int, Hq: int, D: int, window, sinks32, out,
                      scale: Optional[float] = None, kv_heads: Optional[int] = None, table: Optional[torch.Tensor] = None,
                      visible: P.Visible = P.PLAIN) -> None:
        """The streamed paged-attention kernel finishing its rows itself.  Up to 1024 rows take the balanced persistent form
        (every CTA moves the same number of tiles, whatever the rows' lengths); more rows take one CTA per (row, head, chunk)."""
        longest = min(self.max_len, window + visible.keep if window else self.max_len, visible.chunk or self.max_len)
        max_tiles = -(-longest // 64) + 1 + int(visible.keep > 0)         # (+ 1: a window, or kept first keys, that straddle a tile boundary)
        # (factors and sigmoid weights are built for the balanced form)
        persist = visible.gain is not None or visible.sigmoid is not None or (R <= 1024 and os.environ.get("DEWB_DECODE_PERSIST", "1") == "1")
        if persist:
            min_tiles = int(os.environ.get("DEWB_DECODE_MIN_TILES", self.MIN_TILES))
            splits = (max_tiles - 1) // min_tiles + 2
        else:
            share = 8                                                     # tiles a CTA takes
            splits = max(1, -(-max_tiles // share))
        n = R * Hq * splits
        scale = 1.0 / math.sqrt(D) if scale is None else scale
        kv_heads = self.kv_heads if kv_heads is None else kv_heads
        pm, pl, pa = self._partials(n, D, q.device)
        if getattr(self, "_arrivals", None) is None or self._arrivals.numel() < R * kv_heads:
            self._arrivals = torch.zeros(R * kv_heads, dtype=torch.int32, device=q.device)
        common = (L.ptr(q), L.ptr(self.k[layer]), L.ptr(self.v[layer]), ctypes.c_longlong(self.pages * self.page_size),
                  L.ptr(self.page_table if table is None else table), L.ptr(lens32), L.ptr(pm), L.ptr(pl), L.ptr(pa), L.ptr(self._arrivals), L.ptr(sinks32),
                  L.ptr(out), ctypes.c_int(R), ctypes.c_int(Hq), ctypes.c_int(kv_heads), ctypes.c_int(self.page_size),
                  ctypes.c_int(self.max_pages), ctypes.c_int(splits))
        if persist:
            if getattr(self, "_ctas", None) is None:
                self._ctas = 2 * torch.cuda.get_device_properties(q.device).multi_processor_count
            L.check(lib.dewb_paged_decode_persist(*common, ctypes.c_int(min_tiles), ctypes.c_float(scale),
                                                  ctypes.c_int(window or 0), ctypes.c_int(visible.keep), ctypes.c_int(visible.chunk or 0),
                                                ctypes.c_float(visible.softcap), L.ptr(visible.gain), L.ptr(visible.sigmoid), ctypes.c_longlong(q_row_stride),
                                                ctypes.c_int(self._ctas),
                                                  L.ptr(L.status(q.device)), L.stream_ptr()), "paged_decode_persist")
        else:
            L.check(lib.dewb_paged_decode_fused(*common, ctypes.c_int(share), ctypes.c_float(scale),
                                                ctypes.c_int(window or 0), ctypes.c_int(visible.keep), ctypes.c_int(visible.chunk or 0),
                                                ctypes.c_float(visible.softcap), ctypes.c_longlong(q_row_stride),
                                                L.ptr(L.status(q.device)), L.stream_ptr()), "paged_decode_fused")
        L.count_launches()

    def decode_packed(self, layer: int, qkv: torch.Tensor, cos, sin, positions: torch.Tensor, Hq: int, window=None, sinks=None):
        """One decode step of a layer straight from the packed projection output ``qkv [R, Hq + 2 Hkv, D]``: one kernel rotates
        the query / key heads in place and appends the keys and values to the paged cache, then the streamed paged-attention
        kernel reads the queries where they are (row stride of the packed tensor).  Returns ``[R, Hq, D]``."""
        lib = L.load()
        R, H, D = qkv.shape
        pos32, lens32 = self._step_ints(positions)
        L.check(lib.dewb_rope_append(L.ptr(qkv), L.ptr(cos), L.ptr(sin), L.ptr(pos32), ctypes.c_int(R), ctypes.c_int(Hq),
                                     ctypes.c_int(self.kv_heads), ctypes.c_int(D), ctypes.c_int(cos.shape[0] if cos is not None else 0),
                                     L.ptr(self.k[layer]), L.ptr(self.v[layer]), L.ptr(self.page_table), ctypes.c_int(self.page_size),
                                     ctypes.c_int(self.max_pages), L.stream_ptr()), "rope_append")
        out = torch.empty((R, Hq, D), dtype=qkv.dtype, device=qkv.device)
        sk = getattr(self, "_sinks32", None)
        if sinks is not None and (sk is None or sk[0] is not sinks):
            self._sinks32 = sk = (sinks, sinks.detach().float().contiguous())
        self._fused_decode(lib, layer, qkv, H * D, lens32, R, Hq, D, window, sk[1] if sinks is not None else None, out)
        L.count_launches(1)
        return out

    # ------------------------------------------------------------------ reads
    def gather(self, layer: int, length: int, dtype=None) -> Tuple[torch.Tensor, torch.Tensor]:
        """Dense ``[R, length, Hkv, D]`` views of the selected rows' first ``length`` cached tokens."""
        R = self.rows if self.row_ids is None else self.row_ids.numel()
        rows = self._rows(R)[:, None].expand(R, length)
        pos = torch.arange(length, device=self.device)[None].expand(R, length)
        slots = self._slots(rows.reshape(-1), pos.reshape(-1))
        kp = self.k[layer].reshape(-1, self.kv_heads, self.head_dim)[slots]
        vp = self.v[layer].reshape(-1, self.kv_heads, self.head_dim)[slots]
        dt = dtype or self.dtype
        if self.kind:
            kp = dequantize(kp, self.k_scale[layer].reshape(-1, self.kv_heads)[slots], dt)
            vp = dequantize(vp, self.v_scale[layer].reshape(-1, self.kv_heads)[slots], dt)
        shape = (R, length, self.kv_heads, self.head_dim)
        return kp.reshape(shape).to(dt), vp.reshape(shape).to(dt)

    def decode_attention(self, layer: int, q: torch.Tensor, lengths: torch.Tensor, scale=None, window=None, sinks=None,
                         softcap: float = 0.0) -> torch.Tensor:
        """``q [R, Hq, D]`` against each row's first ``lengths[r]`` cached tokens -> ``[R, Hq, D]``."""
        R, Hq, D = q.shape
        scale = scale if scale is not None else 1.0 / math.sqrt(D)
        if (L.use_cuda(q) and q.dtype == torch.bfloat16 and self.row_ids is None and R == self.rows and not softcap
                and Hq // self.kv_heads <= 8 and D in (64, 128, 256)):
            lib = L.load()
            splits = 1
            longest = self.max_len
            while splits < 16 and R * self.kv_heads * splits < 592 and longest // (splits * 2) >= 256:
                splits *= 2
            # a warp walks its keys 32 at a time with a few dependent memory round trips per step: keep a CTA's share of
            # the longest possible row near 512 keys so that the walk is short and there are CTAs to overlap
            splits = max(splits, min(16, (longest + 511) // 512))
            n = R * Hq * splits
            pm, pl, pa = self._partials(n, D, q.device)
            out = torch.empty_like(q)
            qc, lens32 = q.contiguous(), lengths.to(torch.int32).contiguous()      # kept referenced across the launches below
            sinks32 = sinks.float().contiguous() if sinks is not None else None
            if (self.kind == 0 and D == 128 and self.page_size % 64 == 0 and hasattr(lib, "dewb_paged_decode_stream")
                    and os.environ.get("DEWB_DECODE", "stream") == "stream"):
                if scale == 1.0 / math.sqrt(D) and os.environ.get("DEWB_DECODE_FUSED", "1") == "1":
                    self._fused_decode(lib, layer, qc, 0, lens32, R, Hq, D, window, sinks32, out)
                    return out
                # streamed form: TMA page tiles into a shared-memory ring, scores and values on the warp-level tensor cores
                L.check(lib.dewb_paged_decode_stream(L.ptr(qc), L.ptr(self.k[layer]), L.ptr(self.v[layer]),
                                                     ctypes.c_longlong(self.pages * self.page_size), L.ptr(self.page_table), L.ptr(lens32),
                                                     L.ptr(pm), L.ptr(pl), L.ptr(pa), ctypes.c_int(R), ctypes.c_int(Hq),
                                                     ctypes.c_int(self.kv_heads), ctypes.c_int(self.page_size), ctypes.c_int(self.max_pages),
                                                     ctypes.c_int(splits), ctypes.c_float(scale), ctypes.c_int(window or 0), ctypes.c_int(0),
                                                     ctypes.c_int(0), ctypes.c_float(0.0), ctypes.c_longlong(0), L.ptr(L.status(q.device)), L.stream_ptr()), "paged_decode_stream")
                L.check(lib.dewb_decode_combine(L.ptr(pm), L.ptr(pl), L.ptr(pa), L.ptr(sinks32),
                                                L.ptr(out), L.ptr(None), ctypes.c_int(R), ctypes.c_int(Hq), ctypes.c_int(D), ctypes.c_int(splits),
                                                L.stream_ptr()), "decode_combine")
                L.count_launches(2)
                return out
            L.check(lib.dewb_paged_decode(L.ptr(qc), L.ptr(self.k[layer]), L.ptr(self.v[layer]),
                                          L.ptr(self.k_scale[layer] if self.kind else None),
                                          L.ptr(self.v_scale[layer] if self.kind else None), L.ptr(self.page_table),
                                          L.ptr(lens32), L.ptr(sinks32), L.ptr(out), L.ptr(None),
                                          L.ptr(pm), L.ptr(pl), L.ptr(pa), ctypes.c_int(R), ctypes.c_int(Hq),
                                          ctypes.c_int(self.kv_heads), ctypes.c_int(1), ctypes.c_int(D), ctypes.c_int(self.page_size),
                                          ctypes.c_int(self.max_pages), ctypes.c_int(splits), ctypes.c_float(scale),
                                          ctypes.c_int(window or 0), ctypes.c_int(0), ctypes.c_int(0), ctypes.c_float(0.0), L.ptr(None), L.ptr(None), ctypes.c_int(self.kind),
                                          L.stream_ptr()), "paged_decode")
            L.count_launches(2)
            return out
        return paged_attention_reference(self, layer, q, lengths, scale, window, sinks, softcap)

    # ------------------------------------------------------------------ the call attention layers make
    def attend(self, layer: int, q, k, v, positions, causal=True, window=None, softcap=0.0, sinks=None):
        """Write this call's keys / values, then attend. ``q [R, S, Hq, D]``, ``k, v [R, S, Hkv, D]``, ``positions [R, S]``
        (absolute; -1 marks padding). S == 1 is the decode step (paged kernel); S > 1 is a prefill chunk."""
        R, S = q.shape[0], q.shape[1]
        if positions is None:
            positions = torch.arange(S, device=q.device)[None].expand(R, S)
        if S == 1:
            pos = positions[:, 0]
            self.append(layer, k[:, 0], v[:, 0], pos)
            lengths = torch.where(pos >= 0, pos + 1, torch.zeros_like(pos))
            return self.decode_attention(layer, q[:, 0], lengths, window=window, sinks=sinks, softcap=softcap)[:, None]

        self.write(layer, k, v, positions)
        if self.chunk_span is not None:
            # the caller knows where this chunk starts and ends (a server batching rows by start offset): no device read
            start, total, fresh = self.chunk_span[0], self.chunk_span[1], self.chunk_span[0] == 0
        else:
            start = int(positions[:, 0].clamp_min(0).min())
            fresh = start == 0 and bool((positions[:, 0] <= 0).all())
            total = None
        if fresh:
            return ops.attention(q, k, v, causal=causal, window=window, softcap=softcap, sinks=sinks)
        if total is None:
            total = int(positions.max()) + 1
        kc, vc = self.gather(layer, total, dtype=q.dtype)
        # bottom-right aligned causal attention of the chunk against everything cached so far (rows share `start`)
        return ops.attention_reference(q, kc, vc, causal=causal, window=window, softcap=softcap, sinks=sinks)


class Uncached:
    """Stands where a cache would in a forward call over whole sequences: ``attend_slot`` in plain differentiable form, remembering the keys
    and values that later layers read."""
    uncached = True

    def __init__(self, slots: Sequence[CacheSlot]):
        self.slots = list(slots)
        self.sources = {s.source for s in slots if s.source is not None}
        self.source_of = [s.source for s in slots]
        self.kept: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = {}

    def attend_slot(self, slot: int, qkv, heads: P.Heads, positions, *, scale: float, eps: float = 1e-6, q_weight=None, k_weight=None, temperature=None,
                    bias=None, chunk: Optional[int] = None, sinks=None, window: Optional[int] = None, keep: int = 0, softcap: float = 0.0,
                    rot: Optional[rotary.Rotary] = None, unit: bool = False, gain=None, sigmoid=None) -> torch.Tensor:
        R, S, _ = qkv.shape
        pos = torch.arange(S, device=qkv.device)[None].expand(R, S) if positions is None else positions
        turned = None if rot is None else P.Turned(rot, rotary.angles_reference(pos, rot))
        q, k, v = P.prepare_reference(qkv, heads, q_weight, k_weight, eps, temperature, pos, bias, turned, unit)
        if not heads.own:
            k, v = self.kept[self.source_of[slot]]
        elif slot in self.sources:
            self.kept[slot] = (k, v)
        # chunks counted from the first position: documents of the packed-segment form, with ids that start at 1
        segments = None if not chunk else (torch.arange(S, device=qkv.device, dtype=torch.int32) // chunk + 1)[None].expand(R, S).contiguous()
        if (keep and window) or gain is not None or sigmoid is not None:
            o = visible_attention(q, k, v, scale, P.Visible(chunk, sinks, window, keep, softcap, gain, sigmoid))
        else:
            o = ops.attention(q, k, v, causal=True, scale=scale, sinks=sinks, segment_ids=segments, window=window, softcap=softcap)
        return P.head_gate_reference(o, qkv[..., heads.packed:] if heads.gated else None, heads.dv)

    def attend_latent(self, slot: int, z, queries, up, lat: M.Latent, positions, *, scale: float, eps: float, q_weight=None, kv_weight=None,
                      gated: bool = False) -> torch.Tensor:
        R, S, _ = z.shape
        pos = torch.arange(S, device=z.device)[None].expand(R, S) if positions is None else positions
        table = rotary.angles_reference(pos, lat.rotary)
        cq, made = M.prepare_reference(z, lat, q_weight, kv_weight, eps, table)
        q = queries(cq).view(R, S, lat.heads, lat.width)
        q = torch.cat([q[..., :lat.dim], rotary.turn(q[..., lat.dim:], table, lat.rotary).to(q.dtype)], -1)
        wk, wv = lat.split_up(up)
        k = torch.einsum("rsl,hdl->rshd", made.c, wk)
        k = torch.cat([k, made.key.unsqueeze(2).expand(R, S, lat.heads, lat.rot_dim)], -1)
        o = ops.attention(q, k, torch.einsum("rsl,hvl->rshv", made.c, wv), causal=True, scale=scale)
        return M.gate_reference(o.reshape(R, S, lat.heads * lat.vdim), z[..., lat.q_rank + lat.row:] if gated else None)


def visible_attention(q, k, v, scale: float, visible: P.Visible) -> torch.Tensor:
    """Causal attention over whole rows as ``visible`` limits it: ``q [R, S, H, dk]``, ``k, v [R, S, G, *]`` (plain, differentiable)."""
    R, S, H, _ = q.shape
    k, v = (t.float().repeat_interleave(H // t.shape[2], 2) for t in (k, v))
    seen = P.seen_keys(torch.arange(S, device=q.device)[None].expand(R, S), S, visible)
    return torch.einsum("rhsn,rnhd->rshd", P.weights_of(torch.einsum("rshd,rnhd->rhsn", q.float(), k) * scale, seen, visible), v).to(q.dtype)


def paged_attention_reference(store: KVStore, layer: int, q, lengths, scale, window=None, sinks=None, softcap=0.0):
    """fp32 oracle of the paged decode kernel."""
    R, Hq, D = q.shape
    Lmax = max(int(lengths.max()), 1)
    kc, vc = store.gather(layer, Lmax, dtype=torch.float32)
    rep = Hq // store.kv_heads
    kc, vc = kc.repeat_interleave(rep, 2), vc.repeat_interleave(rep, 2)
    s = torch.einsum("rhd,rthd->rht", q.float(), kc) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    t = torch.arange(Lmax, device=q.device)[None, None]
    mask = t < lengths[:, None, None]
    if window:
        mask = mask & (t >= (lengths[:, None, None] - window))
    s = s.masked_fill(~mask, float("-inf"))
    if sinks is not None:
        p = torch.softmax(torch.cat([s, sinks.float().reshape(1, Hq, 1).expand(R, Hq, 1)], -1), -1)[..., :-1]
    else:
        p = torch.softmax(s, -1)
    p = torch.nan_to_num(p)
    return torch.einsum("rht,rthd->rhd", p, vc).to(q.dtype)
