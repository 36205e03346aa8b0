"""Ragenex checkpoints <-> ``CausalTransformer``: static hyper-connections over fp32 streams, layer norms, layer scale, learned positions,
attention without rotation (q / k norms over all heads, a query temperature) beside lightning attention, clamped-GLU feed-forwards, and a
looped block of layers.  ``config.json`` describes every layer by itself, so sizes and constants may differ from layer to layer.

The projections are fused here (q | k | v, gate | up); ``export_state`` takes them apart again.
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Tuple

import torch

from ..models.causal_transformer import CausalTransformer, Loop, TransformerConfig
from .layouts import copy_tensors

ARCHITECTURE = "Ragenex"
KINDS = {"attention": "nope", "lightning": "lightning"}


def is_ragenex(cfg: Mapping[str, Any]) -> bool:
    return str(cfg.get("architecture") or "").lower() == ARCHITECTURE.lower()


def _layer(entry: Mapping[str, Any]) -> Tuple[str, Dict[str, Any], bool]:
    """(mixer kind, layer options, whether it has a feed-forward) of one entry of ``layers``."""
    kind, m, mlp = entry["type"], entry["mixer"], entry.get("mlp")
    if kind not in KINDS:
        raise ValueError(f"unknown mixer {kind!r}; known: {sorted(KINDS)}")
    out: Dict[str, Any] = {"num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m.get("vdim") or m["dim"])}
    if kind == "attention":
        temp = m.get("q_temp")
        out.update(num_kv_heads=int(m.get("kv_heads") or m["heads"]), query_scale=float(m["scale"]),
                   query_temperature=None if not temp else (float(temp["coef"]), int(temp["every"])))
    else:
        out["decay"] = list(m["decay"]) if isinstance(m["decay"], (list, tuple)) else float(m["decay"])
    if mlp:
        if mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: dense")
        out.update(mlp_features=int(mlp["ff"]), mlp_limit=float(mlp["limit"]))
    return KINDS[kind], out, bool(mlp)


def read_ragenex_config(cfg: Mapping[str, Any]) -> TransformerConfig:
    kinds, options, mlps = zip(*(_layer(e) for e in cfg["layers"]))
    loop = cfg.get("loop")
    if loop and (int(loop.get("times", 1)) == 1 or int(loop["stop"]) <= int(loop["start"])):
        loop = None
    return TransformerConfig(
        vocab_size=int(cfg["vocab"]), emb_features=int(cfg["width"]), num_layers=len(kinds), num_heads=options[0]["num_heads"], num_kv_heads=1,
        head_dim=options[0]["head_dim"], max_seq_len=int(cfg["max_positions"]), norm_eps=float(cfg["norm"]["eps"]), qk_norm=False, qk_norm_full=True,
        tie_embeddings=False, norm="layer", layer_types=kinds, layer_options=options, layer_mlp=mlps, mlp_activation="clamped_glu",
        hyper_connections=int(cfg.get("streams") or 1), hyper_dynamic=False, layer_scale=True, learned_positions=True,
        loop=None if not loop else Loop(steps=int(loop["times"]), first=int(loop["start"]), end=int(loop["stop"])))


def ragenex(dtype=None, device=None, **fields) -> CausalTransformer:
    """A freshly initialised model from the fields of a ``config.json`` (the registry's name for the design)."""
    model = CausalTransformer(read_ragenex_config(fields), dtype=dtype, device=device)
    model.family = "ragenex"
    return model


def write_ragenex_config(c: TransformerConfig) -> Dict[str, Any]:
    names = {v: k for k, v in KINDS.items()}
    layers = []
    mlps = c.layer_mlp if c.layer_mlp is not None else (True,)
    for i, kind in enumerate(c.kinds()):
        l = c.of_layer(i)
        has_mlp = bool(mlps[i % len(mlps)])
        if kind == "lightning":
            o = l.mixer_options
            mixer: Dict[str, Any] = {"heads": o["num_heads"], "dim": o["head_dim"], "vdim": o.get("value_dim", o["head_dim"]), "decay": o["decay"]}
        else:
            hd = l.head_dim or l.emb_features // l.num_heads
            mixer = {"heads": l.num_heads, "kv_heads": l.num_kv_heads or l.num_heads, "dim": hd, "vdim": l.value_dim or hd,
                     "scale": hd ** -0.5 if l.query_scale is None else l.query_scale}
            if l.query_temperature is not None:
                mixer["q_temp"] = {"coef": l.query_temperature[0], "every": l.query_temperature[1]}
        layers.append({"type": names[kind], "mixer": mixer,
                       "mlp": {"kind": "dense", "ff": l.mlp_features, "limit": l.mlp_limit} if has_mlp else None})
    out = {"architecture": ARCHITECTURE, "vocab": c.vocab_size, "width": c.emb_features, "max_positions": c.max_seq_len, "norm": {"eps": c.norm_eps},
           "streams": c.hyper_connections, "layers": layers}
    if c.loop is not None:
        out["loop"] = {"start": c.loop.first, "stop": c.num_layers if c.loop.end is None else c.loop.end, "times": c.loop.steps}
    return out


def _tensors(model: CausalTransformer) -> List[Tuple[torch.Tensor, Tuple[str, ...]]]:
    """Every parameter with the release's tensors that make it up, joined along their first axis."""
    out: List[Tuple[torch.Tensor, Tuple[str, ...]]] = [(model.embed.weight, ("embed",)), (model.position_embed.weight, ("pos",))]
    for i, layer in enumerate(model.layers):
        pre = f"l{i}."
        m, mix = layer.mixer, f"{pre}mix."
        out.append((layer.input_norm.weight, (pre + "norm1",)))
        if layer.kind == "lightning":
            out += [(m.qkv.weight, (mix + "q", mix + "k", mix + "v")), (m.output_gate.weight, (mix + "g",)), (m.norm_weight, (mix + "norm",)),
                    (m.out_proj.weight, (mix + "o",))]
        else:
            out += [(m.qkv_proj.weight, (mix + "q", mix + "k", mix + "v")), (m.q_norm.weight, (mix + "q.norm",)), (m.k_norm.weight, (mix + "k.norm",)),
                    (m.o_proj.weight, (mix + "o",))]
        if layer.mlp is not None:
            out += [(layer.post_norm.weight, (pre + "norm2",)), (layer.mlp.gate_up_proj.weight, (pre + "mlp.gate", pre + "mlp.up")),
                    (layer.mlp.down_proj.weight, (pre + "mlp.down",))]
        for q, (connection, scale) in enumerate(zip(layer.streams, layer.layer_scale), start=1):
            out += [(scale, (f"{pre}ls{q}",)), (connection.alpha, (f"{pre}hc{q}.in",)), (connection.beta, (f"{pre}hc{q}.out",)),
                    (connection.mix, (f"{pre}hc{q}.mix",))]
    return out + [(model.final_norm.weight, ("final.norm",)), (model.head.weight, ("head",))]


def _without_feed_forward(model: CausalTransformer) -> Tuple[str, ...]:
    """Prefixes a layer without a feed-forward has no use for (a release may store them all the same)."""
    return tuple(f"l{i}.{name}" for i, layer in enumerate(model.layers) if layer.mlp is None for name in ("norm2", "ls2", "hc2.", "mlp."))


def load_ragenex_state(model: CausalTransformer, tensors: Mapping[str, torch.Tensor], strict: bool = True) -> List[str]:
    """Copy a release's tensors into ``model``; returns the names nothing read (raises on them with ``strict``)."""
    return copy_tensors(_tensors(model), tensors, strict, _without_feed_forward(model))


def export_ragenex_state(model: CausalTransformer) -> Dict[str, torch.Tensor]:
    """The model's tensors under the release's names."""
    out: Dict[str, torch.Tensor] = {}
    for p, names in _tensors(model):
        t = p.detach()
        if len(names) == 1:
            out[names[0]] = t
        elif len(names) == 2:
            out[names[0]], out[names[1]] = t.chunk(2, 0)
        else:
            layer = model.layers[int(names[0][1:].split(".")[0])]
            m = layer.mixer
            dk, dv = (m.h * m.d, m.h * m.dv) if layer.kind == "lightning" else (m.num_heads * m.head_dim, m.num_kv_heads * m.value_dim)
            k = m.h * m.d if layer.kind == "lightning" else m.num_kv_heads * m.head_dim
            out[names[0]], out[names[1]], out[names[2]] = t.split([dk, k, dv], 0)
    return {k: v.contiguous() for k, v in out.items()}
