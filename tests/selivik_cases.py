"""Small random Selivik models for the tests: configurations, and weights drawn so that every mechanism moves the logits."""
import copy
import functools

import torch

import selivik_oracle as O
from fakonex_cases import cut, error, prompt, replay, row_errors, write  # noqa: F401  (schedules and measures of any design)


def attention(heads, kv, dim, vdim, scale, dims=None, window=None, keep=0, cap=None, factor=None, base=500.0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims or dim}}
    if factor:
        m["rot"]["scaling"] = {"factor": factor}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if cap:
        m["softcap"] = cap
    return "attention", m


def latent(heads, dim, rot, vdim, rank, q_rank, scale, base=300.0):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
                                "rot": {"base": base, "dims": rot}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def config(width, vocab, layers, embed=3.0, gain=0.6, eps=1e-5):
    """``layers``: ((type, mixer), feed-forward or None) pairs."""
    return {"architecture": "Selivik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed}, "residual_mult": gain,
            "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m), mlp in layers]}


CASES = {
    # part of a head rotating, values of another width than the keys, every feed-forward
    "plain": config(24, 37, [(attention(4, 2, 8, 12, 0.4, 4, 7, 2, 3.0, 2.0), dense(14)), (latent(3, 6, 4, 5, 10, 7, 0.35), experts(5, 2, 9)),
                             (attention(4, 1, 10, 6, 0.3, 10, 12, 5, 2.0, 4.0), experts(4, 1, 8))]),
    # odd sizes, layers without a feed-forward, no window, no cap, no scaling, a window of one, more kept keys than the window holds, all experts chosen
    "odd": config(30, 41, [(latent(5, 7, 2, 9, 11, 13, 0.5), None), (attention(6, 3, 7, 5, 0.5, 6), experts(3, 3, 7)), (attention(3, 3, 9, 11, 0.3, 2, 1, 3, 1.5), None),
                           (attention(6, 2, 5, 5, 0.4, 4, 4, 9, None, 3.0), dense(5)), (latent(2, 3, 6, 1, 5, 3, 0.6, 20.0), experts(9, 4, 11))], embed=1.0, gain=1.0, eps=1e-3),
    # one head of everything, a window that keeps nothing
    "single": config(20, 50, [(attention(1, 1, 12, 12, 0.3, 8, 16, 0, 5.0), experts(12, 5, 6)), (latent(1, 12, 8, 12, 12, 12, 0.2), dense(12))], embed=4.5, gain=0.25),
    # widths the tensor-core kernels take (padded to 64 and 128), more than eight query heads per key head, windows across page borders, latent heads of
    # two and three sub-tiles, more than 16 of them
    "wide": config(64, 61, [(attention(12, 1, 40, 40, 0.2, 24, 64, 3, 10.0, 2.0), experts(8, 3, 48)), (latent(5, 64, 32, 64, 96, 40, 0.1), dense(96)),
                            (attention(4, 2, 96, 72, 0.15, 96, 100, 70, 6.0), None), (latent(3, 128, 64, 128, 64, 32, 0.08), experts(6, 2, 40)),
                            (latent(20, 48, 16, 40, 56, 24, 0.12), experts(4, 2, 16)), (attention(8, 2, 128, 128, 0.1, 32, 129, 1, 20.0, 8.0), dense(32))]),
    # windows throughout: nothing past them reaches a token but through the kept ones
    "sealed": config(32, 43, [(attention(4, 2, 16, 16, 0.3, 8, 6, 2, 4.0), experts(6, 2, 12))]),
}


def all_chosen(cfg):
    """The same sizes with every expert chosen: no router call is close in any precision."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rand = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    d = cfg["width"]
    w = {"embed": rand(cfg["vocab"], d), "final.norm": rand(d, std=0.3), "head": rand(cfg["vocab"], d, std=4 * d ** -0.5)}
    for i, layer in enumerate(cfg["layers"]):
        pre, m, mix, mlp = f"l{i}.", layer["mixer"], f"l{i}.mix.", layer["mlp"]
        w[pre + "norm1"], w[pre + "ls1"] = rand(d, std=0.3), 1 + rand(d, std=0.3)
        H, dv = m["heads"], m["vdim"]
        if layer["type"] == "attention":
            for name, rows in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * dv)):
                w[mix + name], w[mix + name + ".b"] = rand(rows, d, std=d ** -0.5), rand(rows, std=0.5)
            w[mix + "sink"] = rand(H) + 1
        else:
            rq, rk, wide = m["q_rank"], m["kv_rank"], m["dim"] + m["rot_dim"]
            w[mix + "dq"], w[mix + "dq.norm"], w[mix + "uq"] = rand(rq, d, std=d ** -0.5), 1 + rand(rq, std=0.3), rand(H * wide, rq, std=2 * rq ** -0.5)
            w[mix + "dkv"], w[mix + "dkv.norm"] = rand(rk + m["rot_dim"], d, std=2 * d ** -0.5), 1 + rand(rk, std=0.3)
            w[mix + "uk"], w[mix + "uv"] = rand(H * m["dim"], rk, std=rk ** -0.5), rand(H * dv, rk, std=rk ** -0.5)
            w[mix + "g"] = rand(H * dv, d, std=d ** -0.5)
        w[mix + "o"] = rand(d, H * dv, std=2 * (H * dv) ** -0.5)
        if mlp:
            w[pre + "ls2"] = 1 + rand(d, std=0.3)
            names = [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            for name, n in names:
                w[f"{pre}mlp.{name}gate"], w[f"{pre}mlp.{name}up"] = rand(n, d, std=2 * d ** -0.5), rand(n, d, std=2 * d ** -0.5)
                w[f"{pre}mlp.{name}down"] = rand(d, n, std=n ** -0.5)
            if mlp["kind"] == "moe":
                E = mlp["router"]["experts"]
                w[pre + "mlp.router"], w[pre + "mlp.router.b"] = rand(E, d, std=2 * d ** -0.5), rand(E, std=0.7)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def load(tmp_path, name, dtype=torch.float32, device="cpu", seed=0):
    """(config, tensors, model) of a case, the model loaded from a release directory."""
    from dew_b200.interop.hf import Pretrained
    cfg = CASES[name] if isinstance(name, str) else name
    w = tensors(cfg, seed)
    m = Pretrained.load(write(tmp_path / "model", cfg, w), dtype=dtype, device=device).eval()
    for p in m.parameters():
        p.requires_grad_(False)
    return cfg, w, m


@functools.lru_cache(maxsize=None)
def wanted(name, length, seed=1, sure=False):
    """(tokens, the restated decoder's logits and residuals) of a case."""
    cfg = all_chosen(CASES[name]) if sure else CASES[name]
    tokens = prompt(cfg, length, seed)
    return (tokens,) + O.run(cfg, tensors(cfg), tokens)
