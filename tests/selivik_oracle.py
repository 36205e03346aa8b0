"""A plain, slow restatement of the Selivik decoder on the CPU: one function per mechanism, one token (or one score row) at a time, in double
precision unless told otherwise.  It shares no code with the library and is what the tests of the design compare against.

``run(config, tensors, tokens)`` takes the ``config.json`` mapping, the checkpoint's tensors by name and one sequence, and returns the
logits of every position and the residual after every layer.
"""
import math

import torch

F = torch.float64


def unit(x, eps):
    """``x`` over its root mean square."""
    return x / torch.sqrt((x * x).sum() / x.numel() + eps)


def rms_norm(x, w, eps):
    return unit(x, eps) * w


def centred_norm(x, w, eps):
    """The norm of the residual: weights are stored as their distance from one."""
    return unit(x, eps) * (1 + w)


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def angle(p, i, dims, base, factor=1.0):
    return p * base ** (-2 * i / dims) / factor


def rotate_pairs(x, p, pairs, base, dims, factor=1.0):
    """``x`` with every pair ``(a, b)`` of places (the i-th of ``pairs``) turned by the i-th angle of position ``p``."""
    y = x.clone()
    t = torch.tensor([angle(p, i, dims, base, factor) for i in range(len(pairs))], dtype=F)
    a, b = (torch.tensor([pair[j] for pair in pairs]) for j in range(2))
    y[a], y[b] = (x[a] * t.cos() - x[b] * t.sin()).to(x.dtype), (x[b] * t.cos() + x[a] * t.sin()).to(x.dtype)
    return y


def halves(dims):
    return [(i, i + dims // 2) for i in range(dims // 2)]


def neighbours(dims):
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


def visible(i, size=None, keep=0):
    """The positions that position ``i`` sees."""
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep]


def capped(s, cap):
    return s if not cap else cap * torch.tanh(s / cap)


def sink_softmax(s, sink=None):
    """Weights of the scores ``s`` when the denominator also counts ``exp(sink)`` (None: an ordinary softmax)."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() if sink is None else e.sum() + torch.exp(sink - m))


def attend(qs, ks, vs, scale, cap=None, size=None, keep=0, sinks=None):
    """``qs [T][H, dk]``, ``ks [T][G, dk]``, ``vs [T][G, dv]`` -> ``[T][H, dv]``."""
    out = []
    H, G = qs[0].shape[0], ks[0].shape[0]
    for i in range(len(qs)):
        seen = visible(i, size, keep)
        K, V = torch.stack([ks[j] for j in seen]), torch.stack([vs[j] for j in seen])
        heads = []
        for h in range(H):
            g = h // (H // G)
            heads.append(sink_softmax(capped((K[:, g] @ qs[i][h]) * scale, cap), None if sinks is None else sinks[h]) @ V[:, g])
        out.append(torch.stack(heads))
    return out


def turned_heads(x, heads, p, rot, eps):
    """``[heads * d]`` -> ``[heads, d]``: the first ``dims`` of every head rotated, then the head over its root mean square."""
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    return torch.stack([unit(rotate_pairs(v, p, halves(rot["dims"]), rot["base"], rot["dims"], factor), eps) for v in x.reshape(heads, -1)])


def attention_mixer(hs, w, pre, m, eps):
    proj = lambda n, h: w[pre + n] @ h + w[pre + n + ".b"]
    qs = [turned_heads(proj("q", h), m["heads"], p, m["rot"], eps) for p, h in enumerate(hs)]
    ks = [turned_heads(proj("k", h), m["kv_heads"], p, m["rot"], eps) for p, h in enumerate(hs)]
    vs = [proj("v", h).reshape(m["kv_heads"], m["vdim"]) for h in hs]
    mask = m.get("mask") or {}
    os_ = attend(qs, ks, vs, m["scale"], m.get("softcap"), mask.get("size"), mask.get("keep_first", 0), w[pre + "sink"])
    return [w[pre + "o"] @ o.reshape(-1) for o in os_]


def latent_queries(h, w, pre, m, p, eps):
    """``[heads, dim + rot_dim]``: through their own latent, the last ``rot_dim`` of each head rotated."""
    q = (w[pre + "uq"] @ rms_norm(w[pre + "dq"] @ h, w[pre + "dq.norm"], eps)).reshape(m["heads"], -1)
    rot = m["rot"]
    return torch.stack([torch.cat([v[:m["dim"]], rotate_pairs(v[m["dim"]:], p, neighbours(m["rot_dim"]), rot["base"], rot["dims"])]) for v in q])


def latent_row(h, w, pre, m, p, eps):
    """What a token leaves for later ones: (its normed latent, its rotated key part)."""
    c = w[pre + "dkv"] @ h
    rot = m["rot"]
    return rms_norm(c[:m["kv_rank"]], w[pre + "dkv.norm"], eps), rotate_pairs(c[m["kv_rank"]:], p, neighbours(m["rot_dim"]), rot["base"], rot["dims"])


def latent_mixer(hs, w, pre, m, eps):
    qs = [latent_queries(h, w, pre, m, p, eps) for p, h in enumerate(hs)]
    ks, vs = [], []
    for p, h in enumerate(hs):
        c, turned = latent_row(h, w, pre, m, p, eps)
        k = (w[pre + "uk"] @ c).reshape(m["heads"], m["dim"])
        ks.append(torch.cat([k, turned.expand(m["heads"], -1)], 1))
        vs.append((w[pre + "uv"] @ c).reshape(m["heads"], m["vdim"]))
    os_ = attend(qs, ks, vs, m["scale"])
    return [w[pre + "o"] @ (o.reshape(-1) * sigmoid(w[pre + "g"] @ h)) for o, h in zip(os_, hs)]


def gated_ff(h, w, pre, act):
    return w[pre + "down"] @ (act(w[pre + "gate"] @ h) * (w[pre + "up"] @ h))


def route(z, top):
    """Router logits of one token -> (chosen experts, their weights)."""
    chosen = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    return chosen, sink_softmax(z[chosen])


def feed_forward(h, w, pre, mlp):
    if mlp["kind"] == "dense":
        return gated_ff(h, w, pre, gelu_tanh)
    chosen, weights = route(w[pre + "router"] @ h + w[pre + "router.b"], mlp["router"]["top"])
    return sum(a * gated_ff(h, w, f"{pre}e{e}.", silu) for e, a in zip(chosen, weights))


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer}


def run(config, tensors, tokens, dtype=F):
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, gain = config["norm"]["eps"], config["residual_mult"]
    xs = [w["embed"][t] * config["embedding"]["scale"] for t in tokens]
    after = []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        hs = [centred_norm(x, w[pre + "norm1"], eps) for x in xs]
        ys = [w[pre + "ls1"] * y for y in MIXERS[layer["type"]](hs, w, pre + "mix.", layer["mixer"], eps)]
        if layer.get("mlp"):
            ys = [y + w[pre + "ls2"] * feed_forward(h, w, pre + "mlp.", layer["mlp"]) for y, h in zip(ys, hs)]
        xs = [x + gain * y for x, y in zip(xs, ys)]
        after.append(torch.stack(xs))
    return torch.stack([w["head"] @ centred_norm(x, w["final.norm"], eps) for x in xs]), torch.stack(after)
