"""Small random Rarelorn models for the tests: configurations, and weights drawn so that every mechanism moves the logits."""
import copy
import functools

import torch

import rarelorn_oracle as O
from fakonex_cases import cut, error, prompt, replay, row_errors, write  # noqa: F401  (schedules and measures of any design)


def parallel(heads, kv, dim, vdim, scale, dims, right, conv=4, window=None, cap=None, base=500.0, scales=(0.7, 0.6), rank=6):
    """``right``: (heads, dim).  ``rank`` shows in the tensors alone."""
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "rot": {"base": base, "dims": dims}}
    if window:
        left["mask"] = {"size": window}
    if cap:
        left["softcap"] = cap
    return "parallel", {"left": left, "right": {"heads": right[0], "dim": right[1]}, "left_scale": scales[0], "right_scale": scales[1]}, rank


def mlstm(heads, dim, vdim, cap=6.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, None


def delta(heads, kv, dim, vdim, conv=4):
    return "delta", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, None


def experts(n, top, ff, groups=(1, 1), scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top, "groups": {"count": groups[0], "keep": groups[1]}, "scale": scale}}


RANKS = {}


def config(name, width, vocab, layers, loop=None, eps=1e-5):
    """``layers``: ((type, mixer, rank), feed-forward or None) pairs; ``loop``: (start, stop, times)."""
    cfg = {"architecture": "Rarelorn", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m, _), mlp in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    RANKS[name] = [rank for (_, _, rank), _ in layers]
    cfg["layers"] = copy.deepcopy(cfg["layers"])
    return cfg


CASES = {
    # every mixer, groups, a loop over the first two layers
    "plain": config("plain", 24, 37, [(parallel(4, 2, 8, 12, 0.4, 4, (3, 5), 3, 7, 3.0), experts(6, 2, 9, (3, 2), 1.3)), (mlstm(2, 7, 5), experts(4, 2, 8)),
                                      (delta(4, 2, 6, 9), None)], (0, 2, 2)),
    # odd sizes and taps, layers without a feed-forward, no window, no cap, one tap, every expert chosen, no loop
    "odd": config("odd", 30, 41, [(delta(3, 3, 5, 7, 2), experts(3, 3, 7)), (mlstm(3, 5, 9, 2.0), None), (parallel(6, 3, 7, 5, 0.5, 6, (2, 9), 1, rank=5), None),
                                  (delta(5, 1, 9, 4, 6), experts(10, 3, 6, (5, 3), 0.8)), (parallel(3, 1, 10, 11, 0.3, 10, (5, 3), 2, 1, 1.5, scales=(1.2, 1.0), rank=9), None)],
                  eps=1e-3),
    # three passes over the middle, layers on both sides
    "looped": config("looped", 20, 50, [(delta(2, 1, 8, 8, 3), None), (mlstm(1, 12, 12), experts(4, 1, 8, (2, 1))), (parallel(2, 1, 8, 8, 0.35, 8, (2, 6), 4, 16, 5.0),
                                        experts(8, 3, 6, (4, 2), 2.0)), (mlstm(4, 4, 6), None)], (1, 3, 3)),
    # one pass, which has a vector and restates nothing
    "once": config("once", 16, 33, [(mlstm(2, 6, 6), None), (delta(2, 2, 6, 6), experts(4, 2, 5, (2, 2)))], (1, 2, 1)),
    # widths the tensor-core kernels take (padded to 64, 128 and 256), more than eight query heads per key head, windows across page borders, heads of 64 and
    # 128 key columns
    "wide": config("wide", 64, 61, [(parallel(12, 1, 40, 40, 0.2, 24, (3, 32), 4, 64, 10.0, rank=16), experts(8, 3, 48, (4, 3), 1.5)), (delta(6, 2, 64, 48), None),
                                    (mlstm(3, 64, 80), experts(6, 2, 40)), (parallel(4, 2, 96, 72, 0.15, 96, (2, 64), 4, 100, 6.0, rank=10), None),
                                    (delta(2, 2, 128, 128, 4), None), (parallel(3, 3, 64, 136, 0.15, 32, (1, 128), 2, 129, 20.0, rank=24), experts(4, 2, 16)),
                                    (mlstm(2, 128, 128, 15.0), None)], (1, 3, 2)),
    # attention in a window behind a convolution alone: nothing past their reach gets to a token
    "sealed": config("sealed", 32, 43, [(parallel(4, 2, 16, 16, 0.3, 8, (2, 8), 3, 6, 4.0, scales=(1.5, 0.0)), experts(6, 2, 12, (3, 2)))]),
}


def all_chosen(cfg):
    """The same sizes with every expert chosen: no router call is close in any precision."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"]:
            r = layer["mlp"]["router"]
            r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return cfg


def tensors(cfg, name="plain", seed=0):
    g = torch.Generator().manual_seed(seed)
    rand = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    d = cfg["width"]
    w = {"embed": rand(cfg["vocab"], d), "final.norm": torch.tensor(1.3), "head": rand(cfg["vocab"], d, std=4 * d ** -0.5)}
    if cfg.get("loop"):
        w["loop.step"] = rand(cfg["loop"]["times"], d)
    for i, layer in enumerate(cfg["layers"]):
        pre, m, mix, mlp = f"l{i}.", layer["mixer"], f"l{i}.mix.", layer["mlp"]
        w[pre + "norm1"] = torch.tensor(0.8 + 0.1 * i)
        lin = lambda key, rows, cols=d, std=1.0: w.__setitem__(key, rand(rows, cols, std=std * cols ** -0.5))
        conv = lambda key, rows, taps: w.__setitem__(key, rand(rows, taps, std=taps ** -0.5))
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                lin(f"{mix}left.{n}", rows, std=1.5)
                w[f"{mix}left.{n}.b"] = rand(rows, std=0.5)
                conv(f"{mix}left.{n}.conv", rows, a["conv"])
            w[mix + "left.temp"], w[mix + "left.pb"] = 1 + rand(H, std=0.3), rand(H) - 1
            lin(mix + "left.o", d, H * dv)
            w[mix + "left.o.b"] = rand(d, std=0.5)
            h, rd, rank = r["heads"], r["dim"], RANKS[name][i]
            for n in "rkvgw":
                w[f"{mix}right.mu.{n}"] = torch.rand(d, generator=g)
            for n in "rkvg":
                lin(f"{mix}right.{n}", h * rd)
            lin(mix + "right.w1", rank, std=1.0)
            lin(mix + "right.w2", h * rd, rank, std=1.5)
            w[mix + "right.w0"], w[mix + "right.u"], w[mix + "right.norm"] = rand(h * rd) - 1.5, rand(h, rd), 1 + rand(h * rd, std=0.3)
            lin(mix + "right.o", d, h * rd, std=2)
        else:
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            G = m.get("kv_heads", H)
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv), ("g", H * dv)):
                lin(mix + n, rows)
                if "conv" in m and n != "g":
                    conv(f"{mix}{n}.conv", rows, m["conv"])
            lin(mix + "o", d, H * dv, std=2)
            if layer["type"] == "mlstm":
                w[mix + "norm"] = 1 + rand(H * dv, std=0.3)
                lin(mix + "i", H, std=2)
                lin(mix + "f", H, std=2)
                w[mix + "i.b"], w[mix + "f.b"] = rand(H), rand(H) + 2
            else:
                w[mix + "norm"] = 1 + rand(dv, std=0.3)
                lin(mix + "b", H, std=2)
                lin(mix + "a", H)
                w[mix + "A_log"], w[mix + "dt_bias"] = rand(H) - 1.5, rand(H)
        if mlp:
            w[pre + "norm2"] = torch.tensor(1.1 - 0.1 * i)
            for e in range(mlp["router"]["experts"]):
                n, ff = f"{pre}mlp.e{e}.", mlp["expert"]["ff"]
                lin(n + "gate", ff, std=2)
                lin(n + "up", ff, std=2)
                lin(n + "down", d, ff)
            lin(pre + "mlp.router", mlp["router"]["experts"], std=2)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def load(tmp_path, name, dtype=torch.float32, device="cpu", seed=0, sure=False):
    """(config, tensors, model) of a case, the model loaded from a release directory."""
    from dew_b200.interop.hf import Pretrained
    cfg = all_chosen(CASES[name]) if sure else CASES[name]
    w = tensors(cfg, name, seed)
    m = Pretrained.load(write(tmp_path / "model", cfg, w), dtype=dtype, device=device).eval()
    for p in m.parameters():
        p.requires_grad_(False)
    return cfg, w, m


@functools.lru_cache(maxsize=None)
def wanted(name, length, seed=1, sure=False):
    """(tokens, the restated decoder's logits and residuals) of a case."""
    cfg = all_chosen(CASES[name]) if sure else CASES[name]
    tokens = prompt(cfg, length, seed)
    return (tokens,) + O.run(cfg, tensors(cfg, name), tokens)
