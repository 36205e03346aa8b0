"""Selivik checkpoints <-> ``CausalTransformer``: layers whose mixer and feed-forward read one norm and join an fp32 residual together (layer scales,
a residual factor, norm weights stored around one).  Mixers are softmax attention in a window that keeps the first tokens (rotated halves with linear
scaling, unit norms, a soft cap, a sink per head, biases) and gated latent attention (rotated neighbours); feed-forwards are a GeGLU or a mixture of
SwiGLU experts weighted by the softmax over the chosen logits.  ``config.json`` describes every layer by itself, so sizes and constants may differ
from layer to layer.

The projections are fused here (q | k | v, query latent | latent | key part | gate, keys | values per head, gate | up, the experts stacked);
``export_selivik_state`` takes them apart again.
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Tuple

import torch

from ..models.causal_transformer import CausalTransformer, Mixture, TransformerConfig
from ..nn.mla import MultiHeadLatentAttention
from ..ops.rotary import Rotary
from .layouts import copy_tensors

ARCHITECTURE = "Selivik"
POSITIONS = 1 << 20          # angles are formed from the positions themselves: rows are bounded by the cache alone
KINDS = {"attention": "attention", "latent_attention": "mla"}


def is_selivik(cfg: Mapping[str, Any]) -> bool:
    return str(cfg.get("architecture") or "").lower() == ARCHITECTURE.lower()


def _rotation(rot: Mapping[str, Any], dims: int, interleaved: bool) -> Rotary:
    scaling = rot.get("scaling") or {}
    if scaling.get("kind", scaling.get("type", "linear")) != "linear":
        raise ValueError(f"unknown rotary scaling {scaling}; known: linear (a factor)")
    return Rotary(int(rot.get("dims") or dims), float(rot["base"]), interleaved, float(scaling.get("factor") or 1.0))


def _layer(entry: Mapping[str, Any]) -> Tuple[str, Dict[str, Any], bool]:
    """(mixer kind, layer options, whether it has a feed-forward) of one entry of ``layers``."""
    kind, m, mlp = entry["type"], entry["mixer"], entry.get("mlp")
    if kind not in KINDS:
        raise ValueError(f"unknown mixer {kind!r}; known: {sorted(KINDS)}")
    if kind == "attention":
        mask, dim = m.get("mask") or {}, int(m["dim"])
        out: Dict[str, Any] = {"num_heads": int(m["heads"]), "num_kv_heads": int(m.get("kv_heads") or m["heads"]), "head_dim": dim,
                               "value_dim": int(m.get("vdim") or dim), "query_scale": float(m["scale"]), "attn_softcap": float(m.get("softcap") or 0.0),
                               "window": int(mask.get("size") or 0) or None, "rotation": _rotation(m["rot"], dim, False)}
        out["keep_first"] = int(mask.get("keep_first") or 0) if out["window"] else 0
    else:
        dim, rot_dim = int(m["dim"]), int(m["rot_dim"])
        out = {"num_heads": int(m["heads"]), "mixer_options": {
            "kv_latent": int(m["kv_rank"]), "q_latent": int(m["q_rank"]), "nope_dim": dim, "rope_dim": rot_dim, "v_dim": int(m.get("vdim") or dim),
            "rotation": _rotation(m["rot"], rot_dim, True), "scale": float(m["scale"]), "out_gate": True}}
    if mlp:
        form = mlp.get("kind", "dense")
        if form == "dense":
            out["mlp_features"] = int(mlp["ff"])
        elif form == "moe":
            router = mlp["router"]
            out["mixture"] = Mixture(experts=int(router["experts"]), top_k=int(router["top"]), score_function="top_softmax", router_bias=True,
                                     expert_features=int(mlp["expert"]["ff"]))
        else:
            raise ValueError(f"unknown feed-forward {form!r}; known: dense, moe")
    return KINDS[kind], out, bool(mlp)


def read_selivik_config(cfg: Mapping[str, Any]) -> TransformerConfig:
    kinds, options, mlps = zip(*(_layer(e) for e in cfg["layers"]))
    return TransformerConfig(
        vocab_size=int(cfg["vocab"]), emb_features=int(cfg["width"]), num_layers=len(kinds), num_heads=options[0]["num_heads"], num_kv_heads=1,
        head_dim=options[0].get("head_dim", 8), max_seq_len=POSITIONS, norm_eps=float(cfg["norm"]["eps"]), qk_norm=False, qk_unit_norm=True, qkv_bias=True,
        attention_sinks=True, tie_embeddings=False, fp32_residual=True, parallel_block=True, layer_scale=True, norm_around=1.0, mlp_activation="gelu_tanh",
        embed_multiplier=float((cfg.get("embedding") or {}).get("scale", 1.0)), residual_multiplier=float(cfg.get("residual_mult", 1.0)),
        layer_types=kinds, layer_options=options, layer_mlp=mlps)


def selivik(dtype=None, device=None, **fields) -> CausalTransformer:
    """A freshly initialised model from the fields of a ``config.json`` (the registry's name for the design)."""
    model = CausalTransformer(read_selivik_config(fields), dtype=dtype, device=device)
    model.family = "selivik"
    return model


def write_selivik_config(c: TransformerConfig) -> Dict[str, Any]:
    names = {v: k for k, v in KINDS.items()}
    layers = []
    mlps = c.layer_mlp if c.layer_mlp is not None else (True,)
    for i, kind in enumerate(c.kinds()):
        l = c.of_layer(i)
        rot = l.rotation if kind == "attention" else l.mixer_options["rotation"]
        spec: Dict[str, Any] = {"base": rot.base, "dims": rot.dims}
        if rot.factor != 1.0:
            spec["scaling"] = {"factor": rot.factor}
        if kind == "attention":
            hd = l.head_dim or l.emb_features // l.num_heads
            mixer: Dict[str, Any] = {"heads": l.num_heads, "kv_heads": l.num_kv_heads or l.num_heads, "dim": hd, "vdim": l.value_dim or hd, "rot": spec,
                                     "scale": hd ** -0.5 if l.query_scale is None else l.query_scale}
            if l.attn_softcap:
                mixer["softcap"] = l.attn_softcap
            if l.window:
                mixer["mask"] = {"size": l.window, "keep_first": l.keep_first}
        else:
            o = l.mixer_options
            mixer = {"heads": l.num_heads, "dim": o["nope_dim"], "rot_dim": o["rope_dim"], "vdim": o["v_dim"], "kv_rank": o["kv_latent"],
                     "q_rank": o["q_latent"], "rot": spec, "scale": o["scale"]}
        mlp = None
        if mlps[i % len(mlps)]:
            mix = l.mixture
            mlp = {"kind": "dense", "ff": l.mlp_features} if mix is None else \
                {"kind": "moe", "expert": {"ff": mix.expert_features}, "router": {"experts": mix.experts, "top": mix.top_k}}
        layers.append({"type": names[kind], "mixer": mixer, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "vocab": c.vocab_size, "width": c.emb_features, "norm": {"eps": c.norm_eps},
            "embedding": {"scale": 1.0 if c.embed_multiplier is None else c.embed_multiplier}, "residual_mult": c.residual_multiplier, "layers": layers}


def _tensors(model: CausalTransformer) -> List[Tuple[torch.Tensor, Tuple[str, ...]]]:
    """Every parameter (or slice of one) with the release's tensors that make it up, joined along their first axis."""
    out: List[Tuple[torch.Tensor, Tuple[str, ...]]] = [(model.embed.weight, ("embed",))]
    for i, layer in enumerate(model.layers):
        pre, m = f"l{i}.", layer.mixer
        mix, ff = pre + "mix.", pre + "mlp."
        out += [(layer.input_norm.weight, (pre + "norm1",)), (layer.layer_scale[0], (pre + "ls1",))]
        if isinstance(m, MultiHeadLatentAttention):
            keys, values = m.shape.split_up(m.kv_up.weight)
            out += [(m.in_proj.weight, (mix + "dq", mix + "dkv", mix + "g")), (m.q_norm.weight, (mix + "dq.norm",)), (m.q_up.weight, (mix + "uq",)),
                    (m.kv_norm.weight, (mix + "dkv.norm",)), (keys, (mix + "uk",)), (values, (mix + "uv",))]
        else:
            out += [(m.qkv_proj.weight, tuple(mix + n for n in "qkv")), (m.qkv_proj.bias, tuple(f"{mix}{n}.b" for n in "qkv")), (m.sinks, (mix + "sink",))]
        out.append((m.o_proj.weight, (mix + "o",)))
        if layer.mlp is None:
            continue
        out.append((layer.layer_scale[1], (pre + "ls2",)))
        if layer.sparse:
            e = layer.mlp.experts
            out += [(layer.mlp.router.weight, (ff + "router",)), (layer.mlp.router.logit_bias, (ff + "router.b",))]
            for j in range(e.experts_n):
                out += [(e.gate_up.data[j], (f"{ff}e{j}.gate", f"{ff}e{j}.up")), (e.down.data[j], (f"{ff}e{j}.down",))]
        else:
            out += [(layer.mlp.gate_up_proj.weight, (ff + "gate", ff + "up")), (layer.mlp.down_proj.weight, (ff + "down",))]
    return out + [(model.final_norm.weight, ("final.norm",)), (model.head.weight, ("head",))]


def load_selivik_state(model: CausalTransformer, tensors: Mapping[str, torch.Tensor], strict: bool = True) -> List[str]:
    """Copy a release's tensors into ``model``; returns the names nothing read (raises on them with ``strict``)."""
    # a layer without a feed-forward has no use for its scale, which a release may store all the same
    spare = tuple(f"l{i}.ls2" for i, layer in enumerate(model.layers) if layer.mlp is None)
    return copy_tensors(_tensors(model), tensors, strict, spare)


def _parts(m, names: Tuple[str, ...], rows: int) -> List[int]:
    """Rows of each of the tensors joined in a parameter of ``rows`` rows."""
    if isinstance(m, MultiHeadLatentAttention) and ".mix." in names[0]:
        return [m.shape.q_rank, m.shape.row, m.shape.heads * m.shape.vdim]
    if ".mix." in names[0]:
        H, G, dk, dv = m.heads
        return [H * dk, G * dk, G * dv]
    return [rows // len(names)] * len(names)


def export_selivik_state(model: CausalTransformer) -> Dict[str, torch.Tensor]:
    """The model's tensors under the release's names."""
    out: Dict[str, torch.Tensor] = {}
    for p, names in _tensors(model):
        t = p.detach()
        t = t.flatten(0, 1) if t.dim() == 3 else t
        if len(names) == 1:
            out[names[0]] = t.to(model.embed.weight.dtype)           # (the router's stay in fp32 here)
            continue
        m = model.layers[int(names[0][1:].split(".")[0])].mixer
        out.update(zip(names, t.split(_parts(m, names, t.shape[0]), 0)))
    return {k: v.contiguous() for k, v in out.items()}
