"""A plain, slow restatement of the Ragenex decoder on the CPU: one function per mechanism, one token (or one score row) at a time,
in double precision unless told otherwise.  It shares no code with the library and is what the tests of the design compare against.

``run(config, tensors, tokens)`` takes the ``config.json`` mapping, the checkpoint's tensors by name and one sequence, and returns the
logits of every position and the sum of the residual streams after every layer run.
"""
import math

import torch

F = torch.float64


def layer_norm(x, w, eps):
    mean = x.sum() / x.numel()
    dev = x - mean
    return dev / torch.sqrt((dev * dev).sum() / x.numel() + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).sum() / x.numel() + eps) * w


def silu(x):
    return x / (1 + torch.exp(-x))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


def softmax_attention(qs, ks, vs, scale):
    """``qs [T][H, dk]``, ``ks [T][G, dk]``, ``vs [T][G, dv]`` -> ``[T][H, dv]``; position i sees j <= i."""
    out = []
    H, G = qs[0].shape[0], ks[0].shape[0]
    for i in range(len(qs)):
        K, V = torch.stack(ks[: i + 1]), torch.stack(vs[: i + 1])
        heads = []
        for h in range(H):
            g = h // (H // G)
            s = (K[:, g] @ qs[i][h]) * scale
            e = torch.exp(s - s.max())
            heads.append((e / e.sum()) @ V[:, g])
        out.append(torch.stack(heads))
    return out


def attention_mixer(hs, w, pre, m, eps):
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    qs, ks, vs = [], [], []
    for p, h in enumerate(hs):
        q = rms_norm(w[pre + "q"] @ h, w[pre + "q.norm"], eps)
        k = rms_norm(w[pre + "k"] @ h, w[pre + "k.norm"], eps)
        if m.get("q_temp"):
            q = q * query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"])
        qs.append(q.reshape(H, dk))
        ks.append(k.reshape(G, dk))
        vs.append((w[pre + "v"] @ h).reshape(G, dv))
    return [w[pre + "o"] @ o.reshape(-1) for o in softmax_attention(qs, ks, vs, m["scale"])]


def decayed_recurrence(qs, ks, vs, decay, state=None):
    """``S <- decay S + k v^T``, ``o = S^T q`` per head; returns the outputs and the last state ``[H, dk, dv]``."""
    H, dk = qs[0].shape
    S = torch.zeros(H, dk, vs[0].shape[1], dtype=qs[0].dtype) if state is None else state.clone()
    out = []
    for q, k, v in zip(qs, ks, vs):
        for h in range(H):
            S[h] = decay[h] * S[h] + torch.outer(k[h], v[h])
        out.append(torch.stack([S[h].t() @ q[h] for h in range(H)]))
    return out, S


def lightning_mixer(hs, w, pre, m, eps):
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    qs = [silu(w[pre + "q"] @ h).reshape(H, dk) for h in hs]
    ks = [silu(w[pre + "k"] @ h).reshape(H, dk) for h in hs]
    vs = [silu(w[pre + "v"] @ h).reshape(H, dv) for h in hs]
    os_, _ = decayed_recurrence(qs, ks, vs, m["decay"])
    out = []
    for h, o in zip(hs, os_):
        n = rms_norm(o.reshape(-1), w[pre + "norm"], eps)
        out.append(w[pre + "o"] @ (n / (1 + torch.exp(-(w[pre + "g"] @ h)))))
    return out


def clamped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def feed_forward(h, w, pre, mlp):
    return w[pre + "down"] @ clamped_glu(w[pre + "gate"] @ h, w[pre + "up"] @ h, mlp["limit"])


def stream_read(streams, r):
    return sum(r[s] * streams[s] for s in range(len(streams)))


def stream_write(streams, mix, out, y):
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


def layer_order(config):
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def run(config, tensors, tokens, dtype=F):
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, n = config["norm"]["eps"], config["streams"]
    x = [w["embed"][t] + w["pos"][p] for p, t in enumerate(tokens)]
    streams = [[v.clone() for _ in range(n)] for v in x]
    after = []
    for i in layer_order(config):
        L, pre = config["layers"][i], f"l{i}."
        mixer = {"attention": attention_mixer, "lightning": lightning_mixer}[L["type"]]
        hs = [layer_norm(stream_read(s, w[pre + "hc1.in"]), w[pre + "norm1"], eps) for s in streams]
        ys = mixer(hs, w, pre + "mix.", L["mixer"], eps)
        streams = [stream_write(s, w[pre + "hc1.mix"], w[pre + "hc1.out"], w[pre + "ls1"] * y) for s, y in zip(streams, ys)]
        if L.get("mlp"):
            hs = [layer_norm(stream_read(s, w[pre + "hc2.in"]), w[pre + "norm2"], eps) for s in streams]
            ys = [feed_forward(h, w, pre + "mlp.", L["mlp"]) for h in hs]
            streams = [stream_write(s, w[pre + "hc2.mix"], w[pre + "hc2.out"], w[pre + "ls2"] * y) for s, y in zip(streams, ys)]
        after.append(torch.stack([sum(s) for s in streams]))
    logits = torch.stack([w["head"] @ layer_norm(sum(s), w["final.norm"], eps) for s in streams])
    return logits, torch.stack(after)
