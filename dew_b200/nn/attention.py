"""Self-attention mixer: fused QKV projection, optional QK-norm, RoPE, GQA, sinks / softcap / window, KV cache.

Capability parity: src/dew/nn/mixers/attention.py:984-1764 (``CausalSelfAttention``), src/dew/nn/rope.py.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..ops import paged as P
from ..ops import token_mix
from .layers import Linear, RMSNorm, declare


class SelfAttention(nn.Module):
    def __init__(self, features: int, num_heads: int, num_kv_heads: Optional[int] = None, head_dim: Optional[int] = None,
                 qk_norm: bool = False, bias: bool = False, causal: bool = True, window: Optional[int] = None,
                 softcap: float = 0.0, sinks: bool = False, norm_eps: float = 1e-6, out_zero_init: bool = False,
                 init_std: Optional[float] = None, qkv_bias: bool = False, scale: Optional[float] = None, qk_norm_full: bool = False,
                 out_gate: bool = False, value_dim: Optional[int] = None, temperature=None, chunk: Optional[int] = None, head_gate: bool = False,
                 own_kv: bool = True, rotation=None, keep_first: int = 0, unit_qk: bool = False, conv: int = 0, weighting: str = "softmax",
                 head_temperature: bool = False, dtype=None, device=None):
        super().__init__()
        self.features, self.num_heads = features, num_heads
        # a softmax scale other than head_dim ** -0.5 is folded into the queries (after the norm and the rotation)
        self.q_gain = None if scale is None else float(scale) * (head_dim or features // num_heads) ** 0.5
        self.num_kv_heads = num_kv_heads or num_heads
        self.head_dim = head_dim or features // num_heads
        self.causal, self.window, self.softcap = causal, window, softcap
        self.value_dim = value_dim or self.head_dim
        self.scale = float(scale) if scale is not None else self.head_dim ** -0.5
        # queries grow with the position: (coef, every) multiplies them by 1 + coef ln(floor((p + 1) / every) + 1)
        self.temperature = None if temperature is None else (float(temperature[0]), int(temperature[1]))
        # a query sees no key from before the start of its chunk of positions; head_gate: each head's output times the sigmoid of one number from
        # the layer's input (its rows stand last in the projection); own_kv False: the layer reads another layer's keys and values
        self.chunk, self.head_gate, self.own_kv = chunk, head_gate, own_kv
        # rotation: the layer's own (``ops.rotary.Rotary``) in place of the model's tables; keep_first: keys from the row's start that a window leaves
        # visible; unit_qk: q and k over their root mean square per head, after the rotation and without a weight
        self.rotation, self.keep_first, self.unit_qk = rotation, int(keep_first), unit_qk
        # conv: q, k and v pass a causal convolution of that many taps per channel, behind the projection's bias; weighting 'sigmoid': a visible key weighs
        # the sigmoid of its score plus a number per head, with no sum over the keys; head_temperature: a head's scores times a number of its own
        self.weighting = weighting
        if weighting not in ("softmax", "sigmoid"):
            raise ValueError(f"unknown attention weighting {weighting!r}; known: softmax, sigmoid")
        if weighting == "sigmoid" and sinks:
            raise ValueError("a sink joins a softmax's denominator: sigmoid weights have none")
        if keep_first and window is None:
            raise ValueError("keep_first belongs to a window")
        if unit_qk and (qk_norm or qk_norm_full):
            raise ValueError("q and k pass one norm: qk_norm (weights, in front of the rotation) or unit_qk (none, behind it)")
        if rotation is not None and rotation.dims > self.head_dim:
            raise ValueError(f"a rotation of {rotation.dims} dimensions does not fit heads of {self.head_dim}")
        self.heads = P.Heads(self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, own_kv, head_gate)
        self.qkv_proj = Linear(features, self.heads.row, bias=(bias or qkv_bias) and not head_gate, axes=("embed", "heads"), init_std=init_std, dtype=dtype,
                               device=device)
        # the gates have no bias
        self.heads_bias = declare(nn.Parameter(torch.zeros(self.heads.packed, dtype=dtype, device=device)), ("heads",), "bias") \
            if (bias or qkv_bias) and head_gate else None
        if conv and not (own_kv and not head_gate and causal):
            raise NotImplementedError("a convolution on q, k and v is built for layers with keys and values of their own and without head gates")
        self.conv = None
        if conv:
            from .linear_attention import ShortConv
            self.conv = ShortConv(self.heads.packed, conv, activation=False, dtype=dtype, device=device)
        per_head = lambda there, value: declare(nn.Parameter(torch.full((num_heads,), value, dtype=dtype, device=device)), ("heads",), "scale") if there else None
        self.head_temperature, self.score_bias = per_head(head_temperature, 1.0), per_head(weighting == "sigmoid", 0.0)
        self.o_proj = Linear(self.num_heads * self.value_dim, features, bias=bias, axes=("heads", "embed"),
                             init_std=init_std, zero_init=out_zero_init, dtype=dtype, device=device)
        # Qwen3-Next: the heads' outputs pass a sigmoid gate computed from the layer's input, before the output projection
        self.gate_proj = Linear(features, self.num_heads * self.head_dim, axes=("embed", "heads"), init_std=init_std, dtype=dtype, device=device) if out_gate else None
        # OLMo-2 normalises q and k over all their heads at once (one weight of heads x head_dim); the usual form is per head
        self.qk_norm_full, self.norm_eps = qk_norm_full, norm_eps
        qw, kw = (self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim) if qk_norm_full else (self.head_dim, self.head_dim)
        self.q_norm = RMSNorm(qw, norm_eps, dtype=dtype, device=device) if (qk_norm or qk_norm_full) else None
        self.k_norm = RMSNorm(kw, norm_eps, dtype=dtype, device=device) if (qk_norm or qk_norm_full) and own_kv else None
        self.sinks = declare(nn.Parameter(torch.zeros(num_heads, dtype=dtype, device=device)), ("heads",), "sinks") if sinks else None
        # a layer whose rotary table differs from the model's: (theta, scaling) builds its own; rotary False drops the rotation (NoPE)
        self.rotary, self.own_rope, self._own = rotation is None, None, None
        self.head_transform = None     # a module applied to the heads' outputs [B, S, H, D] before the output projection (dew_b200.nn.dex)
        self.track_qk_max = False      # set by dew_b200.optim.qk_clip.watch: record each head's largest attention logit
        self.qk_max: Optional[torch.Tensor] = None

    def cache_slot(self, source: Optional[int] = None):
        from .kv_cache import CacheSlot
        more = () if self.conv is None or self.conv.kernel_size < 2 else (("conv", (self.heads.packed, self.conv.kernel_size - 1)),)
        return CacheSlot(self.num_kv_heads, self.head_dim, self.value_dim, source=source, more=more)

    @torch.no_grad()
    def _record_qk_max(self, q, k):
        """Per query head, the largest visible logit ``scale * q . k`` of this call (exact, computed in key blocks)."""
        B, S, H, D = q.shape
        T, Hkv = k.shape[1], k.shape[2]
        qf = q.float().reshape(B, S, Hkv, H // Hkv, D)
        best = torch.full((H,), float("-inf"), device=q.device)
        qi = torch.arange(S, device=q.device)[:, None] + (T - S)
        for t0 in range(0, T, 1024):
            kb = k[:, t0:t0 + 1024].float()
            s = torch.einsum("bsgrd,btgd->bgrst", qf, kb) * (D ** -0.5)
            if self.causal:
                s = s.masked_fill(~(torch.arange(t0, t0 + kb.shape[1], device=q.device)[None, :] <= qi), float("-inf"))
            best = torch.maximum(best, s.amax((0, 3, 4)).reshape(H))
        self.qk_max = best if self.qk_max is None else torch.maximum(self.qk_max, best)

    def project(self, x, cos=None, sin=None, positions=None):
        B, S, _ = x.shape
        H, Hkv, D = self.num_heads, self.num_kv_heads, self.head_dim
        qkv = self.qkv_proj(x).view(B, S, H + 2 * Hkv, D)
        if self.q_norm is not None and self.qk_norm_full:
            q = self.q_norm(qkv[:, :, :H].reshape(B, S, H * D)).view(B, S, H, D)
            k = self.k_norm(qkv[:, :, H:H + Hkv].reshape(B, S, Hkv * D)).view(B, S, Hkv, D)
            qkv = torch.cat([q, k, qkv[:, :, H + Hkv:]], 2)
        elif self.q_norm is not None:
            q = self.q_norm(qkv[:, :, :H])
            k = self.k_norm(qkv[:, :, H:H + Hkv])
            qkv = torch.cat([q, k, qkv[:, :, H + Hkv:]], 2)
        if cos is not None:
            qkv = ops.rope(qkv, cos, sin, positions, rot_heads=H + Hkv)
        q = qkv[:, :, :H]
        return (q if self.q_gain is None else q * self.q_gain), qkv[:, :, H:H + Hkv], qkv[:, :, H + Hkv:]

    def _tables(self, cos, sin):
        if not self.rotary:
            return None, None
        if self.own_rope is None or cos is None:
            return cos, sin
        if self._own is None or self._own[0].device != cos.device or self._own[0].shape[0] != cos.shape[0]:
            theta, scaling = self.own_rope
            self._own = ops.rope_tables(cos.shape[0], self.head_dim, theta, cos.device, scaling)
        return self._own

    def _general(self, x, positions, segment_ids, cache, layer):
        """Heads of any widths, the query temperature, chunks, head gates, windows that keep the first keys, layers that share keys and values, and
        caches whose layers differ; a rotation is the layer's own."""
        from .kv_cache import Uncached
        B, S, _ = x.shape
        if self.rotary or self.gate_proj is not None or segment_ids is not None or not self.causal:
            raise NotImplementedError("a query temperature, values of another width, chunks, head gates, kept first keys, shared keys and per-layer caches are "
                                      "built for causal attention without the model's rotary tables, a full-width output gate or packed segments")
        if self.temperature is not None and (self.rotation is not None or self.unit_qk):
            raise NotImplementedError("a query temperature is built for layers without rotation and unit norms")
        qw, eps = (None, self.norm_eps) if self.q_norm is None else (self.q_norm.weight, self.q_norm.eps)
        kw = None if self.k_norm is None else self.k_norm.weight
        # the bias joins in fp32 where the heads are normalised
        qkv = ops.linear(x, self.qkv_proj.weight) if type(self.qkv_proj) is Linear and self.qkv_proj.bias is not None else self.qkv_proj(x)
        bias = self.qkv_proj.bias if type(self.qkv_proj) is Linear and self.qkv_proj.bias is not None else self.heads_bias
        cache = Uncached(()) if cache is None else cache
        if self.conv is not None:
            kept = getattr(cache, "more", None)
            rows = cache.call(positions).rows if kept is not None else None
            qkv, bias = token_mix.conv_tokens(qkv, self.conv.weight, bias, False, rows, None if kept is None else kept[layer].get("conv")), None
        o = cache.attend_slot(layer, qkv, self.heads, positions, scale=self.scale, eps=eps, q_weight=qw, k_weight=kw, temperature=self.temperature,
                              bias=bias, chunk=self.chunk, sinks=self.sinks, window=self.window, keep=self.keep_first, softcap=self.softcap, rot=self.rotation,
                              unit=self.unit_qk, gain=self.head_temperature, sigmoid=self.score_bias)
        return self.o_proj(o.reshape(B, S, self.num_heads * self.value_dim))

    def forward(self, x, cos=None, sin=None, positions=None, segment_ids=None, cache=None, layer: int = 0):
        B, S, _ = x.shape
        if getattr(cache, "slots", None) is not None or self.temperature is not None or self.value_dim != self.head_dim or self.chunk is not None \
                or self.head_gate or not self.own_kv or self.rotation is not None or self.keep_first or self.unit_qk or self.conv is not None \
                or self.weighting != "softmax" or self.head_temperature is not None:
            return self._general(x, positions, segment_ids, cache, layer)
        cos, sin = self._tables(cos, sin)
        if (cache is None and x.is_cuda and cos is not None and self.head_transform is None and self.gate_proj is None and self.q_norm is None and self.window is None and not self.softcap
                and self.sinks is None and segment_ids is None and not self.track_qk_max and self.q_gain is None):
            from ..ops.attn import packed_attention
            H, Hkv, D = self.num_heads, self.num_kv_heads, self.head_dim
            o = packed_attention(self.qkv_proj(x).view(B, S, H + 2 * Hkv, D), cos, sin, positions, H, Hkv, self.causal)
            if o is not None:
                return self.o_proj(o.reshape(B, S, H * D))
        if (cache is not None and S == 1 and self.q_norm is None and self.q_gain is None and positions is not None and cos is not None
                and self.head_transform is None and self.gate_proj is None and hasattr(cache, "decode_packed")):
            # decode step: rotation, cache append and attention straight from the packed projection (no slices, no copies)
            H, Hkv, D = self.num_heads, self.num_kv_heads, self.head_dim
            qkv = self.qkv_proj(x).view(B, H + 2 * Hkv, D)
            if cache.can_decode_packed(qkv, H, self.softcap):
                o = cache.decode_packed(layer, qkv, cos, sin, positions.reshape(-1), H, window=self.window, sinks=self.sinks)
                return self.o_proj(o.reshape(B, 1, H * D))
        q, k, v = self.project(x, cos, sin, positions)
        if self.track_qk_max and cache is None and self.training:
            self._record_qk_max(q, k)
        if cache is None and hasattr(segment_ids, "visible"):
            # rows that share a prefix (dew_b200.data.forked_rows.Forks): a token sees its own document causally and all of its parent
            if self.window is not None or self.softcap or self.sinks is not None or not self.causal:
                raise NotImplementedError("forked rows are built for plain causal attention (no window, soft cap or sinks)")
            from .attention_variants import biased_attention
            o = biased_attention(q, k, v, mask=segment_ids.visible()[:, None])
        elif cache is not None:
            o = cache.attend(layer, q, k, v, positions, causal=self.causal, window=self.window, softcap=self.softcap,
                             sinks=self.sinks)
        else:
            o = ops.attention(q, k, v, causal=self.causal, window=self.window, softcap=self.softcap, sinks=self.sinks,
                              segment_ids=segment_ids)
        if self.head_transform is not None:
            o = self.head_transform(o)
        o = o.reshape(B, S, self.num_heads * self.head_dim)
        if self.gate_proj is not None:
            o = o * torch.sigmoid(self.gate_proj(x).float()).to(o.dtype)
        return self.o_proj(o)
