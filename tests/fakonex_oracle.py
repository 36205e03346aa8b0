"""A plain, slow restatement of the Fakonex decoder on the CPU: one function per mechanism, one token (or one score row) at a time,
in double precision unless told otherwise.  It shares no code with the library and is what the tests of the design compare against.

``run(config, tensors, tokens)`` takes the ``config.json`` mapping, the checkpoint's tensors by name and one sequence, and returns the
logits of every position and the residual after every layer.
"""
import torch

F = torch.float64


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).sum() / x.numel() + eps) * w


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def head_norm(x, heads, w, eps):
    """``[heads * d]`` -> ``[heads, d]``, every head by its own root mean square, one weight for all."""
    return torch.stack([rms_norm(v, w, eps) for v in x.reshape(heads, -1)])


def first_visible(i, chunk):
    """The first position that position ``i`` sees."""
    return 0 if not chunk else i // chunk * chunk


def sink_softmax(s, sink):
    """Weights of the scores ``s`` when the denominator also counts ``exp(sink)`` (None: an ordinary softmax)."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() if sink is None else e.sum() + torch.exp(sink - m))


def chunked_attention(qs, ks, vs, scale, chunk, sinks=None):
    """``qs [T][H, dk]``, ``ks [T][G, dk]``, ``vs [T][G, dv]`` -> ``[T][H, dv]``."""
    out = []
    H, G = qs[0].shape[0], ks[0].shape[0]
    for i in range(len(qs)):
        lo = first_visible(i, chunk)
        K, V = torch.stack(ks[lo: i + 1]), torch.stack(vs[lo: i + 1])
        heads = []
        for h in range(H):
            g = h // (H // G)
            heads.append(sink_softmax((K[:, g] @ qs[i][h]) * scale, None if sinks is None else sinks[h]) @ V[:, g])
        out.append(torch.stack(heads))
    return out


def project(h, w, name):
    return w[name] @ h + w[name + ".b"]


def keys_and_values(hs, w, pre, m, eps):
    return ([head_norm(project(h, w, pre + "k"), m["kv_heads"], w[pre + "k.norm"], eps) for h in hs],
            [project(h, w, pre + "v").reshape(m["kv_heads"], m["vdim"]) for h in hs])


def attention_mixer(hs, w, pre, m, eps, kv):
    qs = [head_norm(project(h, w, pre + "q"), m["heads"], w[pre + "q.norm"], eps) for h in hs]
    mask = m.get("mask") or {}
    os_ = chunked_attention(qs, kv[0], kv[1], m["scale"], mask.get("size"), w[pre + "sink"])
    return [w[pre + "o"] @ (o * sigmoid(w[pre + "g"] @ h)[:, None]).reshape(-1) for o, h in zip(os_, hs)]


def gated_ff(h, w, pre):
    return w[pre + "down"] @ (silu(w[pre + "gate"] @ h) * (w[pre + "up"] @ h))


def route(z, correction, top, groups=None):
    """Router logits of one token -> (chosen experts, their weights)."""
    s = sigmoid(z)
    choice = s + correction
    if groups:
        parts = choice.reshape(groups["count"], -1)
        best = [float(p.sort(descending=True).values[:2].sum()) for p in parts]
        kept = sorted(range(len(best)), key=lambda g: -best[g])[: groups["keep"]]
        choice = torch.cat([p if g in kept else torch.full_like(p, -float("inf")) for g, p in enumerate(parts)])
    chosen = sorted(range(len(choice)), key=lambda e: -float(choice[e]))[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def expert_mixture(h, w, pre, mlp):
    r = mlp["router"]
    chosen, weights = route(w[pre + "router"] @ h, w[pre + "correction"], r["top"], r.get("groups"))
    y = sum(a * gated_ff(h, w, f"{pre}e{e}.") for e, a in zip(chosen, weights))
    if mlp.get("shared"):
        y = y + sigmoid(w[pre + "shared.sg"] @ h) * gated_ff(h, w, pre + "shared.")
    return y


def run(config, tensors, tokens, dtype=F):
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    xs = [w["embed"][t] for t in tokens]
    after, kept = [], {}
    for i, layer in enumerate(config["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        hs = [rms_norm(x, w[pre + "norm1"], eps) for x in xs]
        source = m.get("kv_from")
        kept[i] = kept[source] if source is not None else keys_and_values(hs, w, pre + "mix.", m, eps)
        ys = attention_mixer(hs, w, pre + "mix.", m, eps, kept[i])
        xs = [x + rms_norm(y, w[pre + "norm1b"], eps) for x, y in zip(xs, ys)]
        if layer.get("mlp"):
            ys = [expert_mixture(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.", layer["mlp"]) for x in xs]
            xs = [x + rms_norm(y, w[pre + "norm2b"], eps) for x, y in zip(xs, ys)]
        after.append(torch.stack(xs))
    logits = torch.stack([w["head"] @ rms_norm(x, w["final.norm"], eps) for x in xs])
    cap = config["logit_softcap"]
    return cap * torch.tanh(logits / cap), torch.stack(after)
