"""Rarelorn checkpoints <-> ``CausalTransformer``: a residual in fp32 under RMS norms of one number each, layers of three kinds - windowed attention with
sigmoid weights beside RWKV-6-style time mixing, the matrix memory of xLSTM, the gated delta rule - and mixtures of SwiGLU experts chosen in groups by a
softmax whose scores are the weights; a block of layers may run several times, each pass with a vector of its own and, from the second on, the embedding
output added in front of it.  ``config.json`` describes every layer by itself, so sizes and constants may differ from layer to layer.

The projections are fused here (q | k | v, with the gate where the mixer has one of that width, the gates' logits, the mixes, the experts stacked);
``export_rarelorn_state`` takes them apart again.
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch

from ..models.causal_transformer import CausalTransformer, Loop, Mixture, TransformerConfig
from ..ops.rotary import Rotary
from .layouts import copy_tensors

ARCHITECTURE = "Rarelorn"
POSITIONS = 1 << 20          # angles are formed from the positions themselves: rows are bounded by the cache alone
KINDS = {"parallel": "pair", "mlstm": "mlstm", "delta": "gdn"}
DECAY_RANK = 64              # a model without a checkpoint has no tensor to take the bottleneck's width from


def is_rarelorn(cfg: Mapping[str, Any]) -> bool:
    return str(cfg.get("architecture") or "").lower() == ARCHITECTURE.lower()


def _attention(m: Mapping[str, Any]) -> Dict[str, Any]:
    dim, rot = int(m["dim"]), m["rot"]
    return {"num_heads": int(m["heads"]), "num_kv_heads": int(m.get("kv_heads") or m["heads"]), "head_dim": dim, "value_dim": int(m.get("vdim") or dim),
            "query_scale": float(m["scale"]), "attn_softcap": float(m.get("softcap") or 0.0), "window": int((m.get("mask") or {}).get("size") or 0) or None,
            "rotation": Rotary(int(rot.get("dims") or dim), float(rot["base"])), "attn_conv": int(m.get("conv") or 0), "attn_weighting": "sigmoid",
            "attn_head_temperature": True, "attn_bias": True}


def _mixer(kind: str, m: Mapping[str, Any], rank: Optional[int]) -> Dict[str, Any]:
    if kind == "parallel":
        r = m["right"]
        return {"left": ("attention", _attention(m["left"])),
                "right": ("rwkv6", {"mixer_options": {"num_heads": int(r["heads"]), "head_dim": int(r["dim"]), "decay_rank": rank or DECAY_RANK}}),
                "left_scale": float(m["left_scale"]), "right_scale": float(m["right_scale"])}
    heads, dim = int(m["heads"]), int(m["dim"])
    vdim = int(m.get("vdim") or dim)
    if kind == "mlstm":
        return {"num_heads": heads, "head_dim": dim, "value_dim": vdim, "gate_cap": float(m["gate_cap"])}
    return {"num_k_heads": int(m.get("kv_heads") or heads), "num_v_heads": heads, "head_k_dim": dim, "head_v_dim": vdim, "conv_size": int(m["conv"]), "qk_eps": 1e-6}


def _mixture(mlp: Mapping[str, Any]) -> Mixture:
    if mlp.get("kind", "moe") != "moe":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: moe")
    r = mlp["router"]
    groups = r.get("groups") or {}
    return Mixture(experts=int(r["experts"]), top_k=int(r["top"]), score_function="softmax", norm_topk_prob=False, scaling=float(r.get("scale", 1.0)),
                   groups=int(groups.get("count") or 1), topk_groups=int(groups.get("keep") or 1), group_best=1, group_fill=float("-inf"),
                   expert_features=int(mlp["expert"]["ff"]))


def read_rarelorn_config(cfg: Mapping[str, Any], tensors: Optional[Mapping[str, torch.Tensor]] = None) -> TransformerConfig:
    """``tensors``: the checkpoint's, whose shapes give what the file does not (the width of a time mixer's bottleneck)."""
    kinds, options, mlps = [], [], []
    for i, entry in enumerate(cfg["layers"]):
        kind, mlp = entry["type"], entry.get("mlp")
        if kind not in KINDS:
            raise ValueError(f"unknown mixer {kind!r}; known: {sorted(KINDS)}")
        rank = int(tensors[f"l{i}.mix.right.w1"].shape[0]) if tensors is not None and kind == "parallel" else None
        option: Dict[str, Any] = {"mixer_options": _mixer(kind, entry["mixer"], rank)}
        if mlp:
            option["mixture"] = _mixture(mlp)
        kinds.append(KINDS[kind])
        options.append(option)
        mlps.append(bool(mlp))
    loop = cfg.get("loop")
    if loop and int(loop["stop"]) <= int(loop["start"]):
        loop = None
    return TransformerConfig(
        vocab_size=int(cfg["vocab"]), emb_features=int(cfg["width"]), num_layers=len(kinds), num_heads=1, num_kv_heads=1, head_dim=8, max_seq_len=POSITIONS,
        norm_eps=float(cfg["norm"]["eps"]), qk_norm=False, tie_embeddings=False, fp32_residual=True, norm_one=True, layer_types=tuple(kinds),
        layer_options=tuple(options), layer_mlp=tuple(mlps),
        loop=None if not loop else Loop(steps=int(loop["times"]), first=int(loop["start"]), end=int(loop["stop"]), restate=True, step_vectors=True))


def rarelorn(dtype=None, device=None, **fields) -> CausalTransformer:
    """A freshly initialised model from the fields of a ``config.json`` (the registry's name for the design)."""
    model = CausalTransformer(read_rarelorn_config(fields), dtype=dtype, device=device)
    model.family = "rarelorn"
    return model


def write_rarelorn_config(c: TransformerConfig) -> Dict[str, Any]:
    names = {v: k for k, v in KINDS.items()}
    layers = []
    for i, kind in enumerate(c.kinds()):
        o, mix = c.of_layer(i).mixer_options, c.of_layer(i).mixture
        if kind == "pair":
            a, r = o["left"][1], o["right"][1]["mixer_options"]
            left: Dict[str, Any] = {"heads": a["num_heads"], "kv_heads": a["num_kv_heads"], "dim": a["head_dim"], "vdim": a["value_dim"], "scale": a["query_scale"],
                                    "conv": a["attn_conv"], "rot": {"base": a["rotation"].base, "dims": a["rotation"].dims}}
            if a["attn_softcap"]:
                left["softcap"] = a["attn_softcap"]
            if a["window"]:
                left["mask"] = {"size": a["window"]}
            mixer: Dict[str, Any] = {"left": left, "right": {"heads": r["num_heads"], "dim": r["head_dim"]}, "left_scale": o["left_scale"],
                                     "right_scale": o["right_scale"]}
        elif kind == "mlstm":
            mixer = {"heads": o["num_heads"], "dim": o["head_dim"], "vdim": o["value_dim"], "gate_cap": o["gate_cap"]}
        else:
            mixer = {"heads": o["num_v_heads"], "kv_heads": o["num_k_heads"], "dim": o["head_k_dim"], "vdim": o["head_v_dim"], "conv": o["conv_size"]}
        mlp = None
        if c.layer_mlp is None or c.layer_mlp[i]:
            mlp = {"kind": "moe", "expert": {"ff": mix.expert_features}, "router": {"experts": mix.experts, "top": mix.top_k, "scale": mix.scaling,
                                                                                    "groups": {"count": mix.groups, "keep": mix.topk_groups}}}
        layers.append({"type": names[kind], "mixer": mixer, "mlp": mlp})
    out = {"architecture": ARCHITECTURE, "vocab": c.vocab_size, "width": c.emb_features, "norm": {"eps": c.norm_eps}, "layers": layers}
    if c.loop is not None:
        out["loop"] = {"start": c.loop.first, "stop": c.num_layers if c.loop.end is None else c.loop.end, "times": c.loop.steps}
    return out


def _attention_tensors(m, pre: str):
    H, G, dk, dv = m.heads
    rows = [H * dk, G * dk, G * dv]
    out = [(m.qkv_proj.weight, tuple(pre + n for n in "qkv"), rows), (m.qkv_proj.bias, tuple(f"{pre}{n}.b" for n in "qkv"), rows)]
    if m.conv is not None:
        out.append((m.conv.weight, tuple(f"{pre}{n}.conv" for n in "qkv"), rows))
    return out + [(m.head_temperature, (pre + "temp",), None), (m.score_bias, (pre + "pb",), None), (m.o_proj.weight, (pre + "o",), None),
                  (m.o_proj.bias, (pre + "o.b",), None)]


def _time_tensors(m, pre: str):
    inner = m.h * m.d
    return [(m.mu, tuple(f"{pre}mu.{n}" for n in m.MIXES), [m.features] * 5), (m.rkvg, tuple(pre + n for n in "rkvg"), [inner] * 4),
            (m.decay_in.weight, (pre + "w1",), None), (m.decay_out.weight, (pre + "w2",), None), (m.decay_base, (pre + "w0",), None), (m.bonus, (pre + "u",), None),
            (m.norm_weight, (pre + "norm",), None), (m.out_proj.weight, (pre + "o",), None)]


def _memory_tensors(m, pre: str):
    key, inner = m.h * m.d, m.h * m.dv
    return [(m.in_proj.weight, tuple(pre + n for n in "qkvg"), [key, key, inner, inner]), (m.gate_proj.weight, (pre + "i", pre + "f"), [m.h, m.h]),
            (m.i_bias, (pre + "i.b",), None), (m.f_bias, (pre + "f.b",), None), (m.norm_weight, (pre + "norm",), None), (m.out_proj.weight, (pre + "o",), None)]


def _delta_tensors(m, pre: str):
    rows = [m.key_dim, m.key_dim, m.value_dim]
    return [(m.in_proj_qkvz.weight, tuple(pre + n for n in "qkvg"), rows + [m.value_dim]), (m.in_proj_ba.weight, (pre + "b", pre + "a"), [m.hv, m.hv]),
            (m.conv1d.weight, tuple(f"{pre}{n}.conv" for n in "qkv"), rows), (m.A_log, (pre + "A_log",), None), (m.dt_bias, (pre + "dt_bias",), None),
            (m.norm_weight, (pre + "norm",), None), (m.out_proj.weight, (pre + "o",), None)]


def _tensors(model: CausalTransformer) -> List[Tuple[torch.Tensor, Tuple[str, ...], Optional[List[int]]]]:
    """Every parameter (or slice of one) with the release's tensors that make it up, joined along their first axis, and how many rows each has."""
    out: List[Tuple[torch.Tensor, Tuple[str, ...], Optional[List[int]]]] = [(model.embed.weight, ("embed",), None)]
    if model.pass_vectors is not None:
        out.append((model.pass_vectors, ("loop.step",), None))
    for i, layer in enumerate(model.layers):
        pre, mix, ff = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
        out.append((layer.input_norm.weight, (pre + "norm1",), None))
        if layer.kind == "pair":
            out += _attention_tensors(layer.mixer.left, mix + "left.") + _time_tensors(layer.mixer.right, mix + "right.")
        else:
            out += (_memory_tensors if layer.kind == "mlstm" else _delta_tensors)(layer.mixer, mix)
        if layer.mlp is None:
            continue
        e = layer.mlp.experts
        out += [(layer.post_norm.weight, (pre + "norm2",), None), (layer.mlp.router.weight, (ff + "router",), None)]
        for j in range(e.experts_n):
            out += [(e.gate_up.data[j], (f"{ff}e{j}.gate", f"{ff}e{j}.up"), [e.hidden] * 2), (e.down.data[j], (f"{ff}e{j}.down",), None)]
    return out + [(model.final_norm.weight, ("final.norm",), None), (model.head.weight, ("head",), None)]


def load_rarelorn_state(model: CausalTransformer, tensors: Mapping[str, torch.Tensor], strict: bool = True) -> List[str]:
    """Copy a release's tensors into ``model``; returns the names nothing read (raises on them with ``strict``)."""
    # what a layer without a feed-forward, or a model without a loop, has no use for a release may store all the same
    spare = tuple(f"l{i}.{name}" for i, layer in enumerate(model.layers) if layer.mlp is None for name in ("norm2", "mlp."))
    if model.pass_vectors is None:
        spare += ("loop.step",)
    return copy_tensors([(p, names) for p, names, _ in _tensors(model)], tensors, strict, spare)


def export_rarelorn_state(model: CausalTransformer) -> Dict[str, torch.Tensor]:
    """The model's tensors under the release's names."""
    out: Dict[str, torch.Tensor] = {}
    for p, names, rows in _tensors(model):
        t = p.detach().to(model.embed.weight.dtype)                       # (routers and gate biases stay in fp32 here)
        if rows is None:
            out[names[0]] = t
            continue
        out.update(zip(names, (t.flatten(0, 1) if t.shape[0] != sum(rows) else t).split(rows, 0)))
    return {k: v.contiguous() for k, v in out.items()}
