"""Fakonex checkpoints <-> ``CausalTransformer``: chunked attention without rotation (per-head q / k norms, biases, a sink and a gate per head,
layers that read an earlier layer's keys and values), group-limited mixtures of experts with a gated shared expert, RMS norms before and after
every sub-layer over an fp32 residual, and soft-capped logits.  ``config.json`` describes every layer by itself, so sizes and constants may
differ from layer to layer.

The projections are fused here (q | k | v | gates, gate | up, the experts stacked); ``export_fakonex_state`` takes them apart again.
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Tuple

import torch

from ..models.causal_transformer import CausalTransformer, Mixture, TransformerConfig
from .layouts import copy_tensors

ARCHITECTURE = "Fakonex"
POSITIONS = 1 << 20          # positions enter no score: rows are bounded by the cache alone


def is_fakonex(cfg: Mapping[str, Any]) -> bool:
    return str(cfg.get("architecture") or "").lower() == ARCHITECTURE.lower()


def _mixture(mlp: Mapping[str, Any]) -> Mixture:
    if mlp.get("kind", "moe") != "moe":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: moe")
    router, groups, shared = mlp["router"], mlp["router"].get("groups") or {}, mlp.get("shared") or {}
    return Mixture(experts=int(router["experts"]), top_k=int(router["top"]), score_function="sigmoid", norm_topk_prob=True, bias=True,
                   expert_features=int(mlp["expert"]["ff"]), shared_features=int(shared.get("ff") or 0), shared_gate=bool(shared),
                   groups=int(groups.get("count") or 1), topk_groups=int(groups.get("keep") or 1), group_fill=float("-inf"))


def _layer(entry: Mapping[str, Any]) -> Tuple[Dict[str, Any], bool]:
    """(layer options, whether it has a feed-forward) of one entry of ``layers``."""
    if entry["type"] != "attention":
        raise ValueError(f"unknown mixer {entry['type']!r}; known: attention")
    m, mlp = entry["mixer"], entry.get("mlp")
    out: Dict[str, Any] = {"num_heads": int(m["heads"]), "num_kv_heads": int(m.get("kv_heads") or m["heads"]), "head_dim": int(m["dim"]),
                           "value_dim": int(m.get("vdim") or m["dim"]), "query_scale": float(m["scale"]),
                           "attn_chunk": int((m.get("mask") or {}).get("size") or 0) or None}
    if m.get("kv_from") is not None:
        out["kv_from"] = int(m["kv_from"])
    if mlp:
        out["mixture"] = _mixture(mlp)
    return out, bool(mlp)


def read_fakonex_config(cfg: Mapping[str, Any]) -> TransformerConfig:
    options, mlps = zip(*(_layer(e) for e in cfg["layers"]))
    return TransformerConfig(
        vocab_size=int(cfg["vocab"]), emb_features=int(cfg["width"]), num_layers=len(options), num_heads=options[0]["num_heads"], num_kv_heads=1,
        head_dim=options[0]["head_dim"], max_seq_len=POSITIONS, norm_eps=float(cfg["norm"]["eps"]), qk_norm=True, qkv_bias=True, attention_sinks=True,
        attn_head_gate=True, tie_embeddings=False, logit_softcap=float(cfg.get("logit_softcap") or 0.0), sandwich_norm=True, fp32_residual=True,
        layer_types=("nope",) * len(options), layer_options=options, layer_mlp=mlps)


def fakonex(dtype=None, device=None, **fields) -> CausalTransformer:
    """A freshly initialised model from the fields of a ``config.json`` (the registry's name for the design)."""
    model = CausalTransformer(read_fakonex_config(fields), dtype=dtype, device=device)
    model.family = "fakonex"
    return model


def write_fakonex_config(c: TransformerConfig) -> Dict[str, Any]:
    layers = []
    mlps = c.layer_mlp if c.layer_mlp is not None else (True,)
    for i in range(c.num_layers):
        l = c.of_layer(i)
        hd = l.head_dim or l.emb_features // l.num_heads
        mixer: Dict[str, Any] = {"heads": l.num_heads, "kv_heads": l.num_kv_heads or l.num_heads, "dim": hd, "vdim": l.value_dim or hd,
                                 "scale": hd ** -0.5 if l.query_scale is None else l.query_scale}
        if l.attn_chunk:
            mixer["mask"] = {"size": l.attn_chunk}
        if l.kv_from is not None:
            mixer["kv_from"] = l.kv_from
        mlp = None
        if mlps[i % len(mlps)]:
            mix = l.mixture
            mlp = {"kind": "moe", "expert": {"ff": mix.expert_features}, "router": {"experts": mix.experts, "top": mix.top_k}}
            if mix.groups > 1:
                mlp["router"]["groups"] = {"count": mix.groups, "keep": mix.topk_groups}
            if mix.shared_features:
                mlp["shared"] = {"ff": mix.shared_features}
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "vocab": c.vocab_size, "width": c.emb_features, "norm": {"eps": c.norm_eps}, "logit_softcap": c.logit_softcap,
            "layers": layers}


def _tensors(model: CausalTransformer) -> List[Tuple[torch.Tensor, Tuple[str, ...]]]:
    """Every parameter (or slice of one) with the release's tensors that make it up, joined along their first axis."""
    out: List[Tuple[torch.Tensor, Tuple[str, ...]]] = [(model.embed.weight, ("embed",))]
    for i, layer in enumerate(model.layers):
        pre, m = f"l{i}.", layer.mixer
        mix = pre + "mix."
        own = ("q", "k", "v") if m.own_kv else ("q",)
        out += [(layer.input_norm.weight, (pre + "norm1",)), (layer.mixer_out_norm.weight, (pre + "norm1b",)),
                (m.qkv_proj.weight, tuple(mix + n for n in own) + (mix + "g",)), (m.heads_bias, tuple(f"{mix}{n}.b" for n in own)),
                (m.q_norm.weight, (mix + "q.norm",)), (m.sinks, (mix + "sink",)), (m.o_proj.weight, (mix + "o",))]
        if m.own_kv:
            out.append((m.k_norm.weight, (mix + "k.norm",)))
        if layer.mlp is not None:
            e, ff = layer.mlp.experts, pre + "mlp."
            out += [(layer.post_norm.weight, (pre + "norm2",)), (layer.mlp_out_norm.weight, (pre + "norm2b",)), (layer.mlp.router.weight, (ff + "router",)),
                    (layer.mlp.router.expert_bias, (ff + "correction",))]
            for j in range(e.experts_n):
                out += [(e.gate_up.data[j], (f"{ff}e{j}.gate", f"{ff}e{j}.up")), (e.down.data[j], (f"{ff}e{j}.down",))]
            if layer.mlp.shared is not None:
                s = layer.mlp.shared
                out += [(s.gate_up_proj.weight, (ff + "shared.gate", ff + "shared.up")), (s.down_proj.weight, (ff + "shared.down",)),
                        (layer.mlp.shared_gate.weight, (ff + "shared.sg",))]
    return out + [(model.final_norm.weight, ("final.norm",)), (model.head.weight, ("head",))]


def load_fakonex_state(model: CausalTransformer, tensors: Mapping[str, torch.Tensor], strict: bool = True) -> List[str]:
    """Copy a release's tensors into ``model``; returns the names nothing read (raises on them with ``strict``)."""
    # a layer without a feed-forward has no use for its norms, which a release may store all the same
    spare = tuple(f"l{i}.{name}" for i, layer in enumerate(model.layers) if layer.mlp is None for name in ("norm2", "mlp."))
    return copy_tensors(_tensors(model), tensors, strict, spare)


def export_fakonex_state(model: CausalTransformer) -> Dict[str, torch.Tensor]:
    """The model's tensors under the release's names."""
    out: Dict[str, torch.Tensor] = {}
    for p, names in _tensors(model):
        t = p.detach()
        if len(names) == 1:
            out[names[0]] = t.to(model.embed.weight.dtype)           # (the router's stay in fp32 here)
            continue
        sizes = [t.shape[0] // len(names)] * len(names)
        if ".mix." in names[0]:
            m = model.layers[int(names[0][1:].split(".")[0])].mixer
            H, G, dk, dv = m.heads
            sizes = ([H * dk] + ([G * dk, G * dv] if m.own_kv else []) + [H])[:len(names)]
        out.update(zip(names, t.split(sizes, 0)))
    return {k: v.contiguous() for k, v in out.items()}
