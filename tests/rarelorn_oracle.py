"""A plain, slow restatement of the Rarelorn decoder on the CPU: one function per mechanism, one token (or one score row) at a time, in double
precision unless told otherwise.  It shares no code with the library and is what the tests of the design compare against.

``run(config, tensors, tokens)`` takes the ``config.json`` mapping, the checkpoint's tensors by name and one sequence, and returns the
logits of every position and the residual after every layer run.
"""
import math

import torch

F = torch.float64


def unit(x, eps):
    """``x`` over its root mean square."""
    return x / torch.sqrt((x * x).sum() / x.numel() + eps)


def scalar_norm(x, g, eps):
    """An RMS norm whose weight is one number for all coordinates."""
    return unit(x, eps) * g


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.maximum(x, torch.zeros_like(x)) + torch.log1p(torch.exp(-x.abs()))


def log_sigmoid(x):
    return -softplus(-x)


def capped(z, cap):
    return z if not cap else cap * torch.tanh(z / cap)


def rotate_halves(x, p, dims, base):
    """The first ``dims`` places of ``x`` turned, place ``i`` against place ``i + dims / 2``."""
    y = x.clone()
    for i in range(dims // 2):
        a = p * base ** (-2 * i / dims)
        u, v = x[i], x[i + dims // 2]
        y[i], y[i + dims // 2] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
    return y


def causal_conv(us, w):
    """``us [T][C]``, ``w [C, taps]``: the last column meets the token itself, what lies before the first token is zero."""
    taps = w.shape[1]
    out = []
    for t in range(len(us)):
        y = torch.zeros_like(us[t])
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y = y + w[:, j] * us[s]
        out.append(y)
    return out


def in_window(i, size=None):
    return [j for j in range(i + 1) if size is None or i - j < size]


def sigmoid_attend(qs, ks, vs, scale, temps, biases, cap=None, size=None):
    """``qs [T][H, dk]``, ``ks [T][G, dk]``, ``vs [T][G, dv]`` -> ``[T][H, dv]``: every visible key weighs a sigmoid of its own."""
    H, G = qs[0].shape[0], ks[0].shape[0]
    out = []
    for i in range(len(qs)):
        seen = in_window(i, size)
        K, V = torch.stack([ks[j] for j in seen]), torch.stack([vs[j] for j in seen])
        heads = []
        for h in range(H):
            g = h // (H // G)
            s = capped((K[:, g] @ qs[i][h]) * scale * temps[h], cap)
            heads.append(sigmoid(s + biases[h]) @ V[:, g])
        out.append(torch.stack(heads))
    return out


def attention_mixer(hs, w, pre, m):
    H, G, dk = m["heads"], m["kv_heads"], m["dim"]
    dv = m.get("vdim") or dk
    proj = {}
    for n in "qkv":
        proj[n] = causal_conv([w[pre + n] @ h + w[pre + n + ".b"] for h in hs], w[pre + n + ".conv"])
    rot = m["rot"]
    turned = lambda xs, heads: [torch.stack([rotate_halves(x, p, rot["dims"], rot["base"]) for x in row.reshape(heads, dk)]) for p, row in enumerate(xs)]
    qs, ks, vs = turned(proj["q"], H), turned(proj["k"], G), [v.reshape(G, dv) for v in proj["v"]]
    os_ = sigmoid_attend(qs, ks, vs, m["scale"], w[pre + "temp"], w[pre + "pb"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return [w[pre + "o"] @ o.reshape(-1) + w[pre + "o.b"] for o in os_]


def shifted(hs, mu):
    """Every token's input drawn towards the one before it (zeros in front of the first)."""
    out, before = [], torch.zeros_like(hs[0])
    for h in hs:
        out.append(h + (before - h) * mu)
        before = h
    return out


def channel_decay(x, w1, w2, w0):
    return torch.exp(-torch.exp(w2 @ torch.tanh(w1 @ x) + w0))


def wkv(rs, ks, vs, ws, u):
    """``[T][H, d]`` each and the bonus ``u [H, d]`` -> ``[T][H, d]``: a token reads the state before its own write, and itself through the bonus."""
    H, d = u.shape
    S = torch.zeros(H, d, vs[0].shape[1], dtype=u.dtype)
    out = []
    for r, k, v, g in zip(rs, ks, vs, ws):
        kv = torch.stack([torch.outer(k[h], v[h]) for h in range(H)])
        out.append(torch.stack([(S[h] + u[h][:, None] * kv[h]).t() @ r[h] for h in range(H)]))
        S = g[:, :, None] * S + kv
    return out


def time_mixer(hs, w, pre, m, eps):
    H, d = m["heads"], m["dim"]
    mixed = {n: shifted(hs, w[pre + "mu." + n]) for n in "rkvgw"}
    r, k, v, g = ([w[pre + n] @ x for x in mixed[n]] for n in "rkvg")
    heads = lambda xs: [x.reshape(H, d) for x in xs]
    ws = [channel_decay(x, w[pre + "w1"], w[pre + "w2"], w[pre + "w0"]) for x in mixed["w"]]
    os_ = wkv(heads(r), heads(k), heads(v), heads(ws), w[pre + "u"])
    return [w[pre + "o"] @ (torch.cat([unit(x, eps) for x in o]) * w[pre + "norm"] * silu(z)) for o, z in zip(os_, g)]


def parallel_mixer(hs, w, pre, m, eps):
    left, right = attention_mixer(hs, w, pre + "left.", m["left"]), time_mixer(hs, w, pre + "right.", m["right"], eps)
    return [m["left_scale"] * a + m["right_scale"] * b for a, b in zip(left, right)]


def gated_delta(qs, ks, vs, betas, decays):
    """``qs, ks [T][H, dk]``, ``vs [T][H, dv]``, ``betas, decays [T][H]`` -> ``[T][H, dv]``: decay, write what the key does not hold yet, read."""
    H, dk = qs[0].shape
    S = [torch.zeros(dk, vs[0].shape[1], dtype=vs[0].dtype) for _ in range(H)]
    out = []
    for q, k, v, b, g in zip(qs, ks, vs, betas, decays):
        row = []
        for h in range(H):
            S[h] = g[h] * S[h]
            S[h] = S[h] + torch.outer(k[h], b[h] * (v[h] - S[h].t() @ k[h]))
            row.append(S[h].t() @ q[h])
        out.append(torch.stack(row))
    return out


def on_the_sphere(x):
    return x / torch.sqrt((x * x).sum() + 1e-6)


def delta_mixer(hs, w, pre, m, eps):
    H, G, dk = m["heads"], m["kv_heads"], m["dim"]
    dv = m.get("vdim") or dk
    q, k, v = ([silu(y) for y in causal_conv([w[pre + n] @ h for h in hs], w[pre + n + ".conv"])] for n in "qkv")
    spread = lambda x: torch.stack([on_the_sphere(x.reshape(G, dk)[h // (H // G)]) for h in range(H)])
    betas = [sigmoid(w[pre + "b"] @ h) for h in hs]
    decays = [torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(w[pre + "a"] @ h + w[pre + "dt_bias"])) for h in hs]
    os_ = gated_delta([spread(x) * dk ** -0.5 for x in q], [spread(x) for x in k], [x.reshape(H, dv) for x in v], betas, decays)
    out = []
    for o, h in zip(os_, hs):
        z = silu(w[pre + "g"] @ h).reshape(H, dv)
        out.append(w[pre + "o"] @ torch.cat([unit(o[j], eps) * w[pre + "norm"] * z[j] for j in range(H)]))
    return out


def matrix_memory(qs, ks, vs, ins, forgets):
    """``qs, ks [T][H, dk]``, ``vs [T][H, dv]``, log gates ``[T][H]`` -> ``[T][H, dv]``; the running maximum starts at 0."""
    H, dk = qs[0].shape
    S = [torch.zeros(dk, vs[0].shape[1], dtype=vs[0].dtype) for _ in range(H)]
    n = [torch.zeros(dk, dtype=vs[0].dtype) for _ in range(H)]
    m = [torch.zeros((), dtype=vs[0].dtype) for _ in range(H)]
    out = []
    for q, k, v, i, f in zip(qs, ks, vs, ins, forgets):
        row = []
        for h in range(H):
            top = torch.maximum(f[h] + m[h], i[h])
            keep, take = torch.exp(f[h] + m[h] - top), torch.exp(i[h] - top)
            S[h], n[h], m[h] = keep * S[h] + take * torch.outer(k[h], v[h]), keep * n[h] + take * k[h], top
            row.append(S[h].t() @ q[h] / (torch.maximum((n[h] @ q[h]).abs(), torch.exp(-top)) + 1e-6))
        out.append(torch.stack(row))
    return out


def mlstm_mixer(hs, w, pre, m, eps):
    H, dk, cap = m["heads"], m["dim"], m["gate_cap"]
    dv = m.get("vdim") or dk
    ins = [capped(w[pre + "i"] @ h + w[pre + "i.b"], cap) for h in hs]
    forgets = [log_sigmoid(capped(w[pre + "f"] @ h + w[pre + "f.b"], cap)) for h in hs]
    os_ = matrix_memory([(w[pre + "q"] @ h).reshape(H, dk) * dk ** -0.5 for h in hs], [(w[pre + "k"] @ h).reshape(H, dk) for h in hs],
                        [(w[pre + "v"] @ h).reshape(H, dv) for h in hs], ins, forgets)
    return [w[pre + "o"] @ (torch.cat([unit(x, eps) for x in o]) * w[pre + "norm"] * sigmoid(w[pre + "g"] @ h)) for o, h in zip(os_, hs)]


def gated_ff(h, w, pre):
    return w[pre + "down"] @ (silu(w[pre + "gate"] @ h) * (w[pre + "up"] @ h))


def route(z, top, groups=1, keep=1, scale=1.0):
    """Router logits of one token -> (chosen experts, their weights): the softmax of all, the best groups by their best expert, the best in those."""
    E = len(z)
    e = torch.exp(z - z.max())
    s = e / e.sum()
    per = E // groups
    order = sorted(range(groups), key=lambda g: -float(s[g * per:(g + 1) * per].max()))
    open_ = [x for g in order[:keep] for x in range(g * per, (g + 1) * per)]
    chosen = sorted(open_, key=lambda x: -float(s[x]))[:top]
    return chosen, s[chosen] * scale


def feed_forward(h, w, pre, mlp):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weights = route(w[pre + "router"] @ h, r["top"], groups["count"], groups["keep"], r.get("scale", 1.0))
    return sum(a * gated_ff(h, w, f"{pre}e{e}.") for e, a in zip(chosen, weights))


MIXERS = {"delta": delta_mixer, "parallel": parallel_mixer, "mlstm": mlstm_mixer}


def order(config):
    """``(layer, pass or None)`` in the order the layers run; a pass number stands at the first layer of each pass of the loop."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    inner = range(loop["start"], loop["stop"])
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in inner]
    return out + [(i, None) for i in range(loop["stop"], n)]


def run(config, tensors, tokens, dtype=F):
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    first = [w["embed"][t] for t in tokens]
    xs, after = list(first), []
    for i, begins in order(config):
        if begins is not None:
            if begins > 0:
                xs = [x + e for x, e in zip(xs, first)]
            xs = [x + w["loop.step"][begins] for x in xs]
        layer, pre = config["layers"][i], f"l{i}."
        ys = MIXERS[layer["type"]]([scalar_norm(x, w[pre + "norm1"], eps) for x in xs], w, pre + "mix.", layer["mixer"], eps)
        xs = [x + y for x, y in zip(xs, ys)]
        if layer.get("mlp"):
            xs = [x + feed_forward(scalar_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.", layer["mlp"]) for x in xs]
        after.append(torch.stack(xs))
    return torch.stack([w["head"] @ scalar_norm(x, w["final.norm"], eps) for x in xs]), torch.stack(after)
