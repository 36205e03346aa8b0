"""Small random Ragenex models for the tests: a configuration, weights drawn so that every mechanism moves the logits, and the schedules
(whole prompts, token by token, portions, batches) that the cached paths are checked with."""
import json

import torch

from dew_b200.checkpoints import tensors as TS


def attention(heads, kv, dim, vdim, scale, temp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return "attention", m


def lightning(heads, dim, vdim, decay):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def config(width, vocab, streams, layers, loop=None, eps=1e-5, max_positions=512):
    """``layers``: (mixer, (ff, limit) or None) pairs."""
    out = {"architecture": "Ragenex", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps}, "max_positions": max_positions,
           "layers": [{"type": kind, "mixer": m, "mlp": None if mlp is None else {"kind": "dense", "ff": mlp[0], "limit": mlp[1]}}
                      for (kind, m), mlp in layers]}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CASES = {
    # one stream, one layer of each kind, values of another width than the keys
    "plain": config(24, 37, 1, [(attention(4, 2, 8, 16, 0.4, (0.5, 3)), (20, 0.8)), (lightning(2, 8, 16, [0.5, 0.95]), (28, 2.5))]),
    # three streams, a looped block, a layer without a feed-forward, three query heads per key head, odd widths
    "looped": config(30, 41, 3, [(lightning(3, 6, 10, [0.3, 0.9, 1.0]), (18, 1.5)), (attention(6, 2, 10, 7, 0.3, (0.2, 5)), None),
                                 (attention(3, 3, 5, 5, 0.6), (17, 0.6)), (lightning(1, 4, 4, [0.0]), None)], loop=(1, 3, 3), eps=1e-3),
    # the loop over the first layers, one key head for all, no temperature, the loop's end in the middle
    "front": config(40, 50, 2, [(attention(5, 1, 16, 16, 0.15), (32, 3.0)), (lightning(2, 16, 8, [0.7, 0.99]), (24, 1.0)),
                                (attention(2, 2, 24, 12, 0.1, (0.3, 1)), (16, 7.0))], loop=(0, 2, 2)),
    # widths the tensor-core kernels take (padded to 64 and 128), more than eight query heads per key head
    "wide": config(64, 61, 4, [(attention(12, 1, 40, 40, 0.2, (0.3, 16)), (64, 1.0)), (lightning(4, 48, 64, [0.6, 0.9, 0.97, 0.999]), (48, 1.2)),
                               (attention(4, 2, 96, 72, 0.1), (64, 2.0)), (lightning(2, 72, 24, [0.8, 0.98]), (40, 0.5))], loop=(1, 3, 2)),
}


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    rand = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    near = lambda *s: 1 + 0.3 * torch.randn(*s, generator=g)
    d, n = cfg["width"], cfg["streams"]
    w = {"embed": rand(cfg["vocab"], d), "pos": rand(cfg["max_positions"], d, std=0.5), "final.norm": near(d), "head": rand(cfg["vocab"], d, std=d ** -0.5)}
    for i, layer in enumerate(cfg["layers"]):
        pre, m, mix = f"l{i}.", layer["mixer"], f"l{i}.mix."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        for name, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            w[mix + name] = rand(rows, d, std=d ** -0.5)
        w[mix + "o"] = rand(d, H * dv, std=(H * dv) ** -0.5)
        if layer["type"] == "attention":
            w[mix + "q.norm"], w[mix + "k.norm"] = 2 * near(H * dk), near(G * dk)
        else:
            w[mix + "g"], w[mix + "norm"] = rand(H * dv, d, std=d ** -0.5), near(H * dv)
        subs = 1
        w[pre + "norm1"] = near(d)
        if layer["mlp"]:
            subs, ff = 2, layer["mlp"]["ff"]
            w[pre + "norm2"] = near(d)
            w[pre + "mlp.gate"], w[pre + "mlp.up"] = rand(ff, d, std=2 * d ** -0.5), rand(ff, d, std=2 * d ** -0.5)
            w[pre + "mlp.down"] = rand(d, ff, std=ff ** -0.5)
        for q in range(1, subs + 1):
            w[f"{pre}ls{q}"] = near(d)
            w[f"{pre}hc{q}.in"], w[f"{pre}hc{q}.out"] = rand(n, std=0.4) + 0.6, rand(n, std=0.4) + 0.8
            w[f"{pre}hc{q}.mix"] = 0.8 * torch.eye(n) + rand(n, n, std=0.2)
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


def error(got, want):
    """Largest row-wise rms difference of centred logits, relative to the spread of the wanted ones."""
    got, want = got.double().cpu(), want.double()
    d = (got - want) - (got - want).mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float(d.pow(2).mean(-1).sqrt().max() / scale)


def replay(model, pieces, rows=1, max_len=None, pool_tokens=None):
    """One sequence cut into ``pieces`` through a ``RowBatch``; logits of every position."""
    from dew_b200.sampling.text import RowBatch
    n = sum(len(p) for p in pieces)
    b = RowBatch(model, rows, max_len or n + 1, pool_tokens=pool_tokens)
    return torch.cat([b.feed([p], [list(range(len(p)))]) for p in pieces])


def cut(tokens, size):
    return [tokens[i:i + size] for i in range(0, len(tokens), size)]
