"""The Rarelorn design for ``bench.py --decoder rarelorn``: the design and its closest existing decoder of equal size (rotary attention in a sliding window
and gated-delta-net layers in the other mixers' places, softmax-routed experts, one bf16 residual), and each of the design's kernels beside the like kernel
of the library's other decoders."""
from __future__ import annotations

from typing import Dict, List

import torch

from .decoder_bench import peaks, replayed, timed

SIZES = {
    "d2048": dict(width=2048, heads=16, kv=4, dim=128, window=1024, time_heads=32, time_dim=64, rank=64, mem_heads=16, mem_dim=128, lin=16, lin_kv=8, lin_dim=128,
                  experts=64, top=8, ff=768, groups=8, keep=4, layers=8, vocab=32768),
    "d4096": dict(width=4096, heads=32, kv=8, dim=128, window=1024, time_heads=64, time_dim=64, rank=64, mem_heads=32, mem_dim=128, lin=32, lin_kv=16, lin_dim=128,
                  experts=32, top=4, ff=1536, groups=4, keep=2, layers=8, vocab=32768),
    "d2048h64": dict(width=2048, heads=32, kv=8, dim=64, window=1024, time_heads=32, time_dim=64, rank=64, mem_heads=32, mem_dim=64, lin=16, lin_kv=8, lin_dim=128,
                     experts=64, top=8, ff=768, groups=8, keep=4, layers=8, vocab=32768),
}
CONV = 4


def design(s: dict, max_len: int, device="cuda"):
    """The design at size ``s``: of every four layers one attention beside time mixing, one matrix memory, two gated delta rules."""
    from ..interop.rarelorn import rarelorn
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"], "scale": 1.5, "groups": {"count": s["groups"], "keep": s["keep"]}}}
    left = {"heads": s["heads"], "kv_heads": s["kv"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5, "softcap": 30.0, "mask": {"size": s["window"]},
            "conv": CONV, "rot": {"base": 1e4, "dims": s["dim"] // 2}}
    pair = {"left": left, "right": {"heads": s["time_heads"], "dim": s["time_dim"]}, "left_scale": 0.7, "right_scale": 0.6}
    memory = {"heads": s["mem_heads"], "dim": s["mem_dim"], "vdim": s["mem_dim"], "gate_cap": 15.0}
    delta = {"heads": s["lin"], "kv_heads": s["lin_kv"], "dim": s["lin_dim"], "vdim": s["lin_dim"], "conv": CONV}
    four = [("parallel", pair), ("mlstm", memory), ("delta", delta), ("delta", delta)]
    m = rarelorn(dtype=torch.bfloat16, device=device, vocab=s["vocab"], width=s["width"], norm={"eps": 1e-5},
                 layers=[{"type": four[i % 4][0], "mixer": four[i % 4][1], "mlp": mlp} for i in range(s["layers"])]).eval()
    with torch.no_grad():
        for layer in m.layers:                                   # what bf16 releases hold
            layer.mlp.router.weight.copy_(layer.mlp.router.weight.to(torch.bfloat16).float())
    return m


def closest(s: dict, max_len: int, device="cuda"):
    from ..models.causal_transformer import CausalTransformer, Mixture, TransformerConfig
    return CausalTransformer(TransformerConfig(
        vocab_size=s["vocab"], emb_features=s["width"], num_layers=s["layers"], num_heads=s["heads"], num_kv_heads=s["kv"], head_dim=s["dim"], max_seq_len=max_len,
        norm_eps=1e-5, qk_norm=False, tie_embeddings=False, layer_types=("local", "gdn", "gdn", "gdn"), window=s["window"],
        mixer_options=dict(num_k_heads=s["lin_kv"], num_v_heads=s["lin"], head_k_dim=s["lin_dim"], head_v_dim=s["lin_dim"], conv_size=CONV),
        mixture=Mixture(experts=s["experts"], top_k=s["top"], expert_features=s["ff"])), dtype=torch.bfloat16, device=device).eval()


@torch.no_grad()
def kernels(s: dict, tokens: int, decode_rows: int, context: int, iters: int) -> List[Dict[str, object]]:
    """Each kernel of the design and a like kernel: milliseconds and fraction of the roofline."""
    import torch.nn.functional as F

    from .. import ops
    from ..nn.kv_cache import CacheSlot, KVCache, KVStore
    from ..ops import conv, flash, gdn, moe_serve, paged, recurrence, rotary, scan, streams, token_mix
    from ..ops.routing import route
    pk = peaks()
    rand = lambda *sh: torch.randn(*sh, dtype=torch.bfloat16, device="cuda")
    d, H, G, D, C, L, LG, W = s["width"], s["heads"], s["kv"], s["dim"], s["window"], s["lin"], s["lin_kv"], s["lin_dim"]
    TH, TD, MH, MD, E, k = s["time_heads"], s["time_dim"], s["mem_heads"], s["mem_dim"], s["experts"], s["top"]
    rows: List[Dict[str, object]] = []

    def entry(name, like, fn, nbytes, flops, fn2, nbytes2, flops2):
        line = {"kernel": name, "like": like}
        for tag, f, b, fl in (("", fn, nbytes, flops), ("like_", fn2, nbytes2, flops2)):
            ms = (replayed if name.startswith("decode") else timed)(f, iters)
            line[tag + "ms"] = ms
            line[tag + "of_roofline"] = max(b / pk["bytes"], fl / pk["flops"]) / ms * 1e3
        rows.append(line)

    T = tokens
    S, R = 4096, max(1, T // 4096)
    Hs, y, y2, one, w, x, br = torch.randn(T, 1, d, device="cuda"), rand(T, d), rand(T, d), rand(1)[0], rand(d), rand(T, d), rand(T, d)
    add = lambda: ops.stream_rms_norm(x, br, w, 1e-5)
    step = lambda write, join=None: (lambda: streams.stream_step(Hs, write, None, one, 1e-5, torch.bfloat16, "rms", 0.0, join))
    entry("stream_step (add, norm of one number)", "stream_rms_norm", step(streams.Write(y)), T * d * 12, 0, add, T * d * 8, 0)
    entry("stream_step (two branches, add, norm)", "stream_rms_norm", step(streams.Write(y, gain=0.7, y2=y2, gain2=0.6)), T * d * 14, 0, add, T * d * 8, 0)
    table, ids = rand(s["vocab"], d), torch.randint(0, s["vocab"], (T,), device="cuda")
    entry("stream_step (add, embedding again and a pass's vector, norm)", "stream_rms_norm", step(streams.Write(y), streams.Join(w, table, ids)), T * d * 14, 0, add,
          T * d * 8, 0)
    del Hs, y, y2, table
    # what a token takes from its neighbours
    pos = torch.arange(S, device="cuda", dtype=torch.int32)[None].repeat(R, 1)
    call = token_mix.Rows(pos, torch.full((R,), S, device="cuda", dtype=torch.int32))
    inner, VD = 2 * LG * W + L * W, L * W
    z, wc, tail = rand(R, S, inner + VD), rand(inner, CONV), torch.zeros(R, inner, CONV - 1, device="cuda")
    plain_in = z[..., :inner].contiguous()
    entry("conv_tokens (silu, state kept)", "short_conv", lambda: token_mix.conv_tokens(z[..., :inner], wc, None, True, call, tail), T * inner * 4, 0,
          lambda: conv.short_conv_cuda(plain_in, wc), T * inner * 4, 0)
    x3, mu, before, gu = x.view(R, S, d), rand(5, d), torch.zeros(R, d, device="cuda"), rand(T, 4 * d)
    entry("shift_tokens (five mixes)", "packed_swiglu", lambda: token_mix.shift_tokens(x3, mu, call, before), T * d * 12, 0, lambda: ops.packed_swiglu(gu), T * d * 12, 0)
    del gu, plain_in
    inw = TH * TD
    zr, w2, w0 = torch.randn(T, s["rank"], device="cuda"), rand(inw, s["rank"]), rand(inw)
    entry("low_rank_decay", "product, tanh and exponentials in PyTorch", lambda: token_mix.low_rank_decay(zr, w2, w0), T * inw * 4 + T * s["rank"] * 4, 0,
          lambda: -torch.exp(F.linear(torch.tanh(zr.bfloat16()), w2, w0).float()), T * inw * 4 + T * s["rank"] * 4, 0)
    wg = rand(2 * L, d)
    entry("narrow_product (gates)", "linear, to fp32", lambda: token_mix.narrow_product(x, wg), T * d * 2, 0, lambda: ops.linear(x, wg).float(), T * d * 2, 0)
    # the recurrences over a prompt
    q, kk, v = F.normalize(rand(R, S, L, W), dim=-1), F.normalize(rand(R, S, L, W), dim=-1), rand(R, S, L, W)
    gg, beta = -torch.rand(R, S, L, device="cuda") * 0.1, torch.rand(R, S, L, device="cuda")
    old = lambda: gdn.gated_delta_rule(q, kk, v, gg, beta, None, None)
    per = R * S * L
    chunk_flops = lambda n, a, b: n * (64 * 2 * (a + b) + 4 * a * b)
    gdn_bytes, gdn_flops = per * (W * 8 + 8), per * (64 * 4 * W + 64 * 2 * W + 6 * W * W)
    gates, A, dt = torch.randn(R, S, 2 * L, device="cuda"), torch.randn(L, device="cuda"), torch.randn(L, device="cuda")
    st = torch.zeros(R, L, W, W, device="cuda")
    zq, zk, zv = z[..., :LG * W], z[..., LG * W:2 * LG * W], z[..., 2 * LG * W:inner]
    entry("delta_rule", "gated delta rule (gdn_sm100)", lambda: recurrence.delta_rule(zq, zk, zv, gates, A, dt, L, LG, None, call, st),
          R * S * (inner + VD) * 2 + per * 8, gdn_flops, old, gdn_bytes, gdn_flops)
    mq, mb = rand(R, S, 4 * MH * MD), torch.randn(MH, device="cuda")
    mem = recurrence.Memory(torch.zeros(R, MH, MD, MD, device="cuda"), torch.zeros(R, MH, MD, device="cuda"), torch.zeros(R, MH, device="cuda"))
    mgates = torch.randn(R, S, 2 * MH, device="cuda")
    a, b, c, g = mq.split(MH * MD, -1)
    entry("matrix_memory", "gated delta rule (gdn_sm100)", lambda: recurrence.matrix_memory(a, b, c, mgates, mb, mb, MH, 15.0, None, call, mem),
          R * S * MH * (MD * 8 + 8), chunk_flops(R * S * MH, MD, MD), old, gdn_bytes, gdn_flops)
    tr, tk, tv, lw, tu = rand(R, S, inw), rand(R, S, inw), rand(R, S, inw), -torch.rand(R, S, inw, device="cuda"), rand(TH, TD)
    tst = torch.zeros(R, TH, TD, TD, device="cuda")
    entry("bonus_decay (time mixing)", "gated delta rule (gdn_sm100)", lambda: recurrence.bonus_decay(tr, tk, tv, lw, tu, TH, call, tst), R * S * inw * 12,
          chunk_flops(R * S * TH, TD, TD), old, gdn_bytes, gdn_flops)
    o, zg, nw, ng = rand(R, S, L, W), z[..., inner:], rand(W), rand(T, L, W)
    entry("head_gated_norm", "gated_rms_norm", lambda: token_mix.head_gated_norm(o, zg, nw, 1e-5), T * VD * 6, 0,
          lambda: ops.gated_rms_norm(o.view(T, L, W), ng, nw, 1e-5), T * VD * 6, 0)
    del z, q, kk, v, gg, beta, gates, mq, a, b, c, g, tr, tk, tv, lw, o, zg, ng
    # attention of prompts
    heads, rot = paged.Heads(H, G, D, D), rotary.Rotary(D // 2, 1e4)
    slot = [CacheSlot(G, D, D)]
    store = KVStore(KVCache(page_size=64), 1, R, S, 0, 0, torch.bfloat16, "cuda", slots=slot)
    plain = KVStore(KVCache(page_size=64), 1, R, S, G, D, torch.bfloat16, "cuda")
    qkv = rand(R, S, heads.row)
    bare = qkv.view(R, S, H + 2 * G, D)
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    cos, sin = ops.rope_tables(S, D, 1e4, "cuda")
    pos64, turned = pos.long(), paged.Turned(rot, rotary.angles(pos, rot))

    def rope_write():
        r = ops.rope(bare, cos, sin, pos64, rot_heads=H + G)
        plain.write(0, r[:, :, H:H + G], r[:, :, H + G:], pos64)
    nb = R * S * heads.packed * 2
    entry("head_norm_append with rotation", "rope + cache write", lambda: paged.qk_norm_append(qkv, heads, None, None, 1e-5, None, pos, pages, None, turned),
          2 * nb + R * S * 2 * G * D * 2, 0, rope_write, 2 * nb + R * S * 2 * G * D * 2, 0)
    packed = paged.qk_norm_append(qkv, heads, None, None, 1e-5, None, pos, pages, None, turned)
    q, kk, v = packed[:, :, :H], packed[:, :, H:H + G], packed[:, :, H + G:]
    gain, pb = torch.rand(H, device="cuda") + 0.5, torch.randn(H, device="cuda") - 4
    fl = 4 * D * H * R * sum(min(i + 1, C) for i in range(S))
    entry("flash, window, soft cap, sigmoid weights", "flash, window, soft cap", lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(C, 30.0, gain=gain, sigmoid=pb)),
          0, fl, lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(C, 30.0)), 0, fl)
    at = S // 2
    q2, p2 = packed[:1, at:at + 512, :H].contiguous(), pos[:1, at:at + 512].contiguous()
    kc, vc = plain.gather(0, at + 512)
    fl = 4 * H * D * 512 * C
    visible = paged.Visible(window=C, softcap=30.0, gain=gain, sigmoid=pb)
    entry(f"paged_attend_mma (512 after {at}, sigmoid weights)", "gathered score matrix", lambda: paged.paged_attend(q2, heads, p2, pages, 0.1, visible=visible), 0, fl,
          lambda: ops.attention_reference(q2, kc[:1], vc[:1], window=C), 0, fl)
    del qkv, bare, packed, q, kk, v, store, plain, kc, vc, pages, q2
    torch.cuda.empty_cache()
    # a decode step
    B = decode_rows
    posd, lens = torch.full((B, 1), context, device="cuda", dtype=torch.int32), torch.full((B,), context + 1, device="cuda")
    call = token_mix.Rows(posd, lens.int())
    store = KVStore(KVCache(page_size=64), 1, B, context + 64, 0, 0, torch.bfloat16, "cuda", slots=slot)
    plain = KVStore(KVCache(page_size=64), 1, B, context + 64, G, D, torch.bfloat16, "cuda")
    qkv1, q0 = rand(B, 1, heads.row), rand(B, H, D)
    entry("decode: sigmoid attention (rotation, append, paged)", "decode attention, window", lambda: store.attend_slot(0, qkv1, heads, posd, scale=0.1, window=C, softcap=30.0,
          rot=rot, gain=gain, sigmoid=pb), B * min(C, context + 1) * 2 * G * D * 2, 0, lambda: plain.decode_attention(0, q0, lens, window=C),
          B * min(C, context + 1) * 2 * G * D * 2, 0)
    del store, plain
    x1, tail1, cache1 = rand(B, 1, inner), torch.zeros(B, inner, CONV - 1, device="cuda"), torch.zeros(B, CONV - 1, inner, device="cuda", dtype=torch.bfloat16)
    entry("decode: conv_tokens", "short_conv_step", lambda: token_mix.conv_tokens(x1, wc, None, True, call, tail1), B * inner * (4 + 24) + inner * 8, 0,
          lambda: scan.short_conv_step(x1[:, 0], wc, None, cache1), B * inner * (4 + 12) + inner * 8, 0)
    st, st2 = torch.zeros(B, L, W, W, device="cuda"), torch.zeros(B, L, W, W, device="cuda")
    gates = torch.randn(B, 1, 2 * L, device="cuda")
    q1, k1, v1 = rand(B, L, W), rand(B, L, W), rand(B, L, W)
    g1, b1 = -torch.rand(B, L, device="cuda"), torch.rand(B, L, device="cuda")
    zq, zk, zv = x1[..., :LG * W], x1[..., LG * W:2 * LG * W], x1[..., 2 * LG * W:]
    old = lambda: scan.gated_delta_rule_step(q1, k1, v1, g1, b1, st2)
    like = B * L * W * W * 8
    entry("decode: delta_rule", "gated_delta_rule_step", lambda: recurrence.delta_rule(zq, zk, zv, gates, A, dt, L, LG, None, call, st), like, 0, old, like, 0)
    a, b, c = rand(B, 1, 3 * MH * MD).split(MH * MD, -1)
    mem = recurrence.Memory(torch.zeros(B, MH, MD, MD, device="cuda"), torch.zeros(B, MH, MD, device="cuda"), torch.zeros(B, MH, device="cuda"))
    mgates = torch.randn(B, 1, 2 * MH, device="cuda")
    entry("decode: matrix_memory", "gated_delta_rule_step", lambda: recurrence.matrix_memory(a, b, c, mgates, mb, mb, MH, 15.0, None, call, mem), B * MH * MD * MD * 8, 0,
          old, like, 0)
    tr, tk, tv, lw = rand(B, 1, inw), rand(B, 1, inw), rand(B, 1, inw), -torch.rand(B, 1, inw, device="cuda")
    tst = torch.zeros(B, TH, TD, TD, device="cuda")
    entry("decode: bonus_decay", "gated_delta_rule_step", lambda: recurrence.bonus_decay(tr, tk, tv, lw, tu, TH, call, tst), B * TH * TD * TD * 8, 0, old, like, 0)
    del st, st2, mem, tst
    xd = rand(B, d)
    entry("decode: narrow_product (gates)", "linear, to fp32", lambda: token_mix.narrow_product(xd, wg), (B + 2 * L) * d * 2, 0, lambda: ops.linear(xd, wg).float(),
          (B + 2 * L) * d * 2, 0)
    # the router
    sel = moe_serve.Selection(E, k, s["groups"], s["keep"], float("-inf"), "softmax", False, 1.5, 1)
    wr = torch.randn(E, d, device="cuda").to(torch.bfloat16).float() * d ** -0.5
    wr = wr.to(torch.bfloat16).float()
    split = moe_serve.split_weights(wr)
    for tag, n in (("router", T), ("decode: router", decode_rows)):
        xs = x[:n].contiguous()
        entry(tag, "fp32 router product + moe_route", lambda: moe_serve.route(xs, wr, split, None, sel), n * d * 2 + E * d * 2, 2 * n * E * d,
              lambda: route(F.linear(xs.float(), wr), None, k, "softmax", True), n * d * 2 + E * d * 4, 2 * n * E * d)
    return rows
