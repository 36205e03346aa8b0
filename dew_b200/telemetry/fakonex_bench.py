"""The Fakonex design for ``bench.py --decoder fakonex``: the design and its closest existing decoder of equal size (rotary attention within a
sliding window as long as the chunks, softmax-routed experts with a shared one, a bf16 residual), and each of the design's kernels beside the
like kernel of that decoder."""
from __future__ import annotations

from typing import Dict, List

import torch

from .decoder_bench import peaks, timed

SIZES = {
    "d2048": dict(width=2048, heads=16, kv=4, dim=128, chunk=2048, experts=64, top=8, groups=8, keep=4, ff=768, shared=768, layers=8, vocab=32768),
    "d4096": dict(width=4096, heads=32, kv=8, dim=128, chunk=2048, experts=32, top=4, groups=4, keep=2, ff=1536, shared=1536, layers=8, vocab=32768),
    "d2048h64": dict(width=2048, heads=32, kv=8, dim=64, chunk=2048, experts=64, top=8, groups=8, keep=4, ff=768, shared=768, layers=8, vocab=32768),
}


def design(s: dict, max_len: int, device="cuda"):
    """The design at size ``s``: every fourth layer reads the keys and values of the one before it."""
    from ..interop.fakonex import fakonex
    layers = []
    for i in range(s["layers"]):
        mixer = {"heads": s["heads"], "kv_heads": s["kv"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5, "mask": {"size": s["chunk"]}}
        if i % 4 == 3:
            mixer["kv_from"] = i - 1
        layers.append({"type": "attention", "mixer": mixer, "mlp": {"kind": "moe", "expert": {"ff": s["ff"]}, "shared": {"ff": s["shared"]},
                       "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}}}})
    m = fakonex(dtype=torch.bfloat16, device=device, vocab=s["vocab"], width=s["width"], norm={"eps": 1e-5}, logit_softcap=30.0, layers=layers).eval()
    with torch.no_grad():
        for layer in m.layers:                                   # what bf16 releases hold
            layer.mlp.router.weight.copy_(layer.mlp.router.weight.to(torch.bfloat16).float())
    return m


def closest(s: dict, max_len: int, device="cuda"):
    from ..models.causal_transformer import CausalTransformer, Mixture, TransformerConfig
    return CausalTransformer(TransformerConfig(
        vocab_size=s["vocab"], emb_features=s["width"], num_layers=s["layers"], num_heads=s["heads"], num_kv_heads=s["kv"], head_dim=s["dim"],
        max_seq_len=max_len, norm_eps=1e-5, qk_norm=False, tie_embeddings=False, layer_types=("local",), window=s["chunk"],
        mixture=Mixture(experts=s["experts"], top_k=s["top"], expert_features=s["ff"], shared_features=s["shared"])), dtype=torch.bfloat16, device=device).eval()


@torch.no_grad()
def kernels(s: dict, tokens: int, decode_rows: int, context: int, iters: int) -> List[Dict[str, object]]:
    """Each kernel of the design and the like kernel of the closest model: milliseconds and fraction of the roofline."""
    import torch.nn.functional as F

    from .. import ops
    from ..nn.kv_cache import CacheSlot, KVCache, KVStore
    from ..ops import moe_serve, paged, streams
    from ..ops import flash
    from ..ops.routing import route
    from ..parallel.ep import TokenExchange
    pk = peaks()
    rand = lambda *sh: torch.randn(*sh, dtype=torch.bfloat16, device="cuda")
    d, H, G, D, C = s["width"], s["heads"], s["kv"], s["dim"], s["chunk"]
    E, k, ff = s["experts"], s["top"], s["ff"]
    rows: List[Dict[str, object]] = []

    def entry(name, like, fn, nbytes, flops, fn2, nbytes2, flops2):
        line = {"kernel": name, "like": like}
        for tag, f, b, fl in (("", fn, nbytes, flops), ("like_", fn2, nbytes2, flops2)):
            ms = timed(f, iters)
            line[tag + "ms"] = ms
            line[tag + "of_roofline"] = max(b / pk["bytes"], fl / pk["flops"]) / ms * 1e3
        rows.append(line)

    T = tokens
    Hs, y, w, x, br = torch.randn(T, 1, d, device="cuda"), rand(T, d), rand(d), rand(T, d), rand(T, d)
    entry("stream_step (norm of the branch, add, norm)", "stream_rms_norm", lambda: streams.stream_step(Hs, streams.Write(y, weight=w, eps=1e-5), None, w, 1e-5,
          torch.bfloat16, "rms"), T * d * 12, 0, lambda: ops.stream_rms_norm(x, br, w, 1e-5), T * d * 8, 0)
    del Hs, y, br
    # attention of prompts: the epilogue of the projection, the attention itself, the gate
    S, R = 4096, max(1, T // 4096)
    heads = paged.Heads(H, G, D, D, True, True)
    slot = [CacheSlot(G, D, D)]
    store = KVStore(KVCache(page_size=64), 1, R, S, 0, 0, torch.bfloat16, "cuda", slots=slot)
    plain = KVStore(KVCache(page_size=64), 1, R, S, G, D, torch.bfloat16, "cuda")
    qkv, pos = rand(R, S, heads.row), torch.arange(S, device="cuda", dtype=torch.int32)[None].repeat(R, 1)
    bare = qkv[..., :heads.packed].contiguous().view(R, S, H + 2 * G, D)
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    qw, kw, bias, sinks = rand(D), rand(D), rand(heads.packed), torch.randn(H, device="cuda")
    cos, sin = ops.rope_tables(S, D, 1e4, "cuda")
    pos64 = pos.long()

    def rope_write():
        r = ops.rope(bare, cos, sin, pos64, rot_heads=H + G)
        plain.write(0, r[:, :, H:H + G], r[:, :, H + G:], pos64)
    nb = R * S * heads.packed * 2
    entry("head_norm_append", "rope + cache write", lambda: paged.qk_norm_append(qkv, heads, qw, kw, 1e-5, None, pos, pages, bias), 2 * nb + R * S * 2 * G * D * 2, 0,
          rope_write, 2 * nb + R * S * 2 * G * D * 2, 0)
    packed = paged.qk_norm_append(qkv, heads, qw, kw, 1e-5, None, pos, pages, bias)
    q, kk, v = packed[:, :, :H], packed[:, :, H:H + G], packed[:, :, H + G:]
    seen = sum(min(i % C, i) + 1 for i in range(S)), sum(min(i + 1, C) for i in range(S))
    entry("flash, chunks and sinks", "flash, window", lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(chunk=C, sinks=sinks)), 0,
          4 * D * H * R * seen[0], lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(window=C)), 0, 4 * D * H * R * seen[1])
    o, gu = q.contiguous(), rand(R * S, 2 * H * D)
    entry("head_gate", "packed_swiglu", lambda: paged.head_gate(o, qkv[..., heads.packed:], D), R * S * H * D * 4, 0, lambda: ops.packed_swiglu(gu),
          R * S * H * D * 6, 0)
    del gu, o
    # a prompt's later portion against what the cache holds (the closest model gathers the pages and forms the score matrix)
    at = min(C + C // 2, S - 512)
    q2, p2 = packed[:1, at:at + 512, :H].contiguous(), pos[:1, at:at + 512].contiguous()
    gate2 = qkv[:1, at:at + 512, heads.packed:]
    fl = 4 * H * D * sum(i % C + 1 for i in range(at, at + 512))
    kc, vc = plain.gather(0, at + 512)
    entry(f"paged_attend_mma (512 after {at})", "gathered score matrix", lambda: paged.paged_attend(q2, heads, p2, pages, 0.1, visible=paged.Visible(C, sinks),
          gate=gate2), 0, fl, lambda: ops.attention_reference(q2, kc[:1], vc[:1], window=C), 0, 4 * H * D * 512 * C)
    del qkv, bare, packed, q, kk, v, store, plain, kc, vc, pages
    # experts: a prompt, then a decode step
    sel = moe_serve.Selection(E, k, s["groups"], s["keep"], float("-inf"), "sigmoid")
    wr, b, gw = torch.randn(E, d, device="cuda").to(torch.bfloat16).float() * d ** -0.5, torch.randn(E, device="cuda") * 0.1, rand(1, d)
    split = moe_serve.split_weights(wr)
    gate_up, down = rand(E, 2 * ff, d) * d ** -0.5, rand(E, d, ff) * ff ** -0.5
    for tag, n in (("prompt", T), ("decode", decode_rows)):
        xs = x[:n].contiguous()
        ex = TokenExchange(E, "self")
        entry(f"router ({tag})", "fp32 router product + moe_route", lambda: moe_serve.route(xs, wr, split, b, sel), n * d * 2 + E * d * 2, 2 * n * E * d,
              lambda: route(F.linear(xs.float(), wr), None, k, "softmax", True), n * d * 2 + E * d * 4, 2 * n * E * d)
        r = moe_serve.route(xs, wr, split, b, sel)
        ids = r.ids.long()
        entry(f"moe_gather ({tag})", "rank + plan + push", lambda: moe_serve.gather(xs, r, gw), n * d * 2 * (1 + k), 0,
              lambda: ex.push(xs, ex.plan(ids, d)), n * d * 2 * (1 + k), 0)
        st = moe_serve.gather(xs, r, gw)
        active = int((r.counts > 0).sum())
        h = moe_serve.product(st.rows, gate_up, st)
        plan = ex.plan(ids, d)
        got = ex.push(xs, plan)
        from ..ops import grouped
        flops, wbytes = 4 * n * k * d * ff, active * 2 * ff * d * 2
        entry(f"grouped product, gate | up ({tag})", "the same after the exchange", lambda: moe_serve.product(st.rows, gate_up, st), wbytes + n * k * (d + 2 * ff) * 2,
              flops, lambda: grouped.gmm_forward(got, gate_up, plan.layout), wbytes + n * k * (d + 2 * ff) * 2, flops)
        entry(f"moe_glu ({tag})", "packed_swiglu on the padded rows", lambda: moe_serve.glu(h, st), n * k * ff * 6, 0, lambda: ops.packed_swiglu(h), n * k * ff * 6, 0)
        a = moe_serve.glu(h, st)
        entry(f"grouped product, down ({tag})", "the same", lambda: moe_serve.product(a, down, st), active * ff * d * 2 + n * k * (d + ff) * 2, flops / 2,
              lambda: moe_serve.product(a, down, st), active * ff * d * 2 + n * k * (d + ff) * 2, flops / 2)
        yy, sh = moe_serve.product(a, down, st), rand(n, d)
        out = torch.empty(ex.rows_cap, d, dtype=torch.bfloat16, device="cuda")

        def pull():
            ex.claim_out(d)
            return ex.pull(ex.claim_out(d), plan, r.weights)[0] + sh
        entry(f"moe_combine with the shared expert ({tag})", "pull + add", lambda: moe_serve.combine(yy, r, st, sh), n * d * 2 * (k + 2), 0, pull, n * d * 2 * (k + 2), 0)
        del ex, h, a, yy, sh, out, st, got, plan
        torch.cuda.empty_cache()
    del gate_up, down, x
    B = decode_rows
    lg, gx = rand(4096, s["vocab"]), rand(4096, s["vocab"])
    entry("softcap (4096 rows of logits)", "packed_swiglu", lambda: streams.softcap(lg, 30.0), lg.numel() * 6, 0, lambda: ops.packed_swiglu(gx), gx.numel() * 3, 0)
    del lg, gx
    store = KVStore(KVCache(page_size=64), 1, B, context + 64, 0, 0, torch.bfloat16, "cuda", slots=slot)
    plain = KVStore(KVCache(page_size=64), 1, B, context + 64, G, D, torch.bfloat16, "cuda")
    q1, lens, posd = rand(B, 1, heads.row), torch.full((B,), context + 1, device="cuda"), torch.full((B, 1), context, device="cuda")
    q0 = q1[..., :heads.packed].reshape(B, H + 2 * G, D)[:, :H].contiguous()
    nb = B * (context % C + 1) * 2 * G * D * 2
    entry("decode attention (norms, append, paged in chunks, gate)", "decode attention, window", lambda: store.attend_slot(0, q1, heads, posd, scale=0.1, eps=1e-5,
          q_weight=qw, k_weight=kw, bias=bias, chunk=C, sinks=sinks), nb, 0, lambda: plain.decode_attention(0, q0, lens, window=C),
          B * min(C, context + 1) * 2 * G * D * 2, 0)
    return rows
