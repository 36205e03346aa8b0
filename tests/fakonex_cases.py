"""Small random Fakonex models for the tests: configurations, weights drawn so that every mechanism moves the logits, and the schedules (whole
prompts, token by token, portions, batches) that the cached paths are checked with."""
import json

import torch

from dew_b200.checkpoints import tensors as TS


def attention(heads, kv, dim, vdim, scale, chunk=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def experts(n, top, ff, shared=None, groups=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(width, vocab, layers, cap=20.0, eps=1e-5):
    """``layers``: (mixer, feed-forward or None) pairs."""
    return {"architecture": "Fakonex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": [{"type": "attention", "mixer": m, "mlp": mlp} for m, mlp in layers]}


CASES = {
    # values of another width than the keys, a layer that reads the first one's keys under a longer chunk of its own
    "plain": config(24, 37, [(attention(4, 2, 8, 16, 0.4, 5), experts(6, 2, 10, 12, (3, 2))),
                             (attention(4, 2, 8, 16, 0.25, 7, kv_from=0), experts(5, 3, 12, 6))]),
    # odd sizes, a layer without a feed-forward, two readers of one layer (one without chunks), three query heads per key head
    "odd": config(30, 41, [(attention(6, 2, 7, 5, 0.5, 11), experts(9, 3, 11, 13, (3, 1))), (attention(3, 3, 5, 9, 0.6, 4), None),
                           (attention(6, 3, 5, 9, 0.4, 9, kv_from=1), experts(4, 1, 9, None, (2, 1))),
                           (attention(3, 3, 5, 9, 0.7, None, kv_from=1), experts(3, 3, 7, 5))], cap=6.0, eps=1e-3),
    # groups of one expert, chunks of one position, one key head for all, more of everything in the last layer
    "single": config(20, 50, [(attention(5, 1, 12, 12, 0.3, 1), experts(4, 1, 8, 8, (4, 2))), (attention(2, 1, 12, 12, 0.3, 16), experts(12, 5, 6, 20, (2, 1)))],
                     cap=40.0),
    # widths the tensor-core kernels take (padded to 64 and 128), more than eight query heads per key head, chunks across page borders
    "wide": config(64, 61, [(attention(12, 1, 40, 40, 0.2, 64), experts(16, 4, 48, 64, (4, 2))), (attention(4, 2, 96, 72, 0.15, 100), experts(8, 2, 40, 24, (2, 1))),
                            (attention(8, 2, 96, 72, 0.1, 128, kv_from=1), experts(8, 3, 64, 32)), (attention(6, 1, 128, 128, 0.1, 48), experts(6, 2, 16, 8, (3, 1)))]),
    # one chunk size throughout: nothing from an earlier chunk reaches a later one
    "sealed": config(32, 43, [(attention(4, 2, 16, 16, 0.3, 6), experts(6, 2, 12, 10, (2, 1))), (attention(4, 4, 8, 8, 0.4, 6), experts(4, 2, 10, 6))]),
}


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rand = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    near = lambda *s: 1 + 0.3 * torch.randn(*s, generator=g)
    d = cfg["width"]
    w = {"embed": rand(cfg["vocab"], d), "final.norm": near(d), "head": rand(cfg["vocab"], d, std=4 * d ** -0.5)}
    for i, layer in enumerate(cfg["layers"]):
        pre, m, mix, mlp = f"l{i}.", layer["mixer"], f"l{i}.mix.", layer["mlp"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            if name == "q" or m.get("kv_from") is None:
                w[mix + name], w[mix + name + ".b"] = rand(rows, d, std=d ** -0.5), rand(rows, std=0.5)
        w[mix + "q.norm"], w[mix + "sink"], w[mix + "g"] = 2 * near(dk), rand(H) + 1, rand(H, d, std=2 * d ** -0.5)
        if m.get("kv_from") is None:
            w[mix + "k.norm"] = near(dk)
        w[mix + "o"] = rand(d, H * dv, std=(H * dv) ** -0.5)
        w[pre + "norm1"], w[pre + "norm1b"] = near(d), near(d)
        if mlp:
            w[pre + "norm2"], w[pre + "norm2b"] = near(d), near(d)
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            # choice scores on both sides of 0: an expert outside the kept groups must not come back in at 0
            w[pre + "mlp.router"], w[pre + "mlp.correction"] = rand(E, d, std=2 * d ** -0.5), rand(E, std=0.4) - 0.9
            for name, n in [(f"e{e}", ff) for e in range(E)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                w[f"{pre}mlp.{name}.gate"], w[f"{pre}mlp.{name}.up"] = rand(n, d, std=2 * d ** -0.5), rand(n, d, std=2 * d ** -0.5)
                w[f"{pre}mlp.{name}.down"] = rand(d, n, std=n ** -0.5)
            if mlp.get("shared"):
                w[pre + "mlp.shared.sg"] = rand(1, d, std=2 * d ** -0.5)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write(directory, cfg, w):
    directory.mkdir(parents=True, exist_ok=True)
    (directory / "config.json").write_text(json.dumps(cfg))
    TS.save_file(w, directory / "model.safetensors")
    return directory


def load(tmp_path, name, dtype=torch.float32, device="cpu", seed=0):
    """(config, tensors, model) of a case, the model loaded from a release directory."""
    from dew_b200.interop.hf import Pretrained
    cfg = CASES[name] if isinstance(name, str) else name
    w = tensors(cfg, seed)
    m = Pretrained.load(write(tmp_path / "model", cfg, w), dtype=dtype, device=device).eval()
    for p in m.parameters():
        p.requires_grad_(False)
    return cfg, w, m


def prompt(cfg, length, seed=1):
    return torch.randint(0, cfg["vocab"], (length,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    """Row-wise rms difference of centred logits, relative to the spread of the wanted ones."""
    got, want = got.double().cpu(), want.double()
    d = (got - want) - (got - want).mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / scale


def error(got, want):
    return float(row_errors(got, want).max())


def replay(model, pieces, rows=1, max_len=None, pool_tokens=None):
    """One sequence cut into ``pieces`` through a ``RowBatch``; logits of every position."""
    from dew_b200.sampling.text import RowBatch
    n = sum(len(p) for p in pieces)
    b = RowBatch(model, rows, max_len or n + 1, pool_tokens=pool_tokens)
    return torch.cat([b.feed([p], [list(range(len(p)))]) for p in pieces])


def cut(tokens, size):
    return [tokens[i:i + size] for i in range(0, len(tokens), size)]
