"""The Selivik design for ``bench.py --decoder selivik``: the design and its closest existing decoder of equal size (rotary attention in a sliding
window and latent attention in the same order, softmax-routed experts, one bf16 residual), and each of the design's kernels beside the like kernel of
the library's other decoders."""
from __future__ import annotations

from typing import Dict, List

import torch

from .decoder_bench import peaks, replayed, timed

SIZES = {
    "d2048": dict(width=2048, heads=16, kv=4, dim=128, window=1024, keep=16, lat_heads=16, lat_dim=128, rot=64, lat_vdim=128, rank=512, q_rank=768, experts=64,
                  top=8, ff=768, dense=5632, layers=8, vocab=32768),
    "d4096": dict(width=4096, heads=32, kv=8, dim=128, window=1024, keep=16, lat_heads=32, lat_dim=128, rot=64, lat_vdim=128, rank=512, q_rank=1536, experts=32,
                  top=4, ff=1536, dense=14336, layers=8, vocab=32768),
    "d2048h64": dict(width=2048, heads=32, kv=8, dim=64, window=1024, keep=16, lat_heads=16, lat_dim=64, rot=32, lat_vdim=64, rank=256, q_rank=512, experts=64,
                     top=8, ff=768, dense=5632, layers=8, vocab=32768),
}


def design(s: dict, max_len: int, device="cuda"):
    """The design at size ``s``: every fourth layer windowed attention, the others latent attention; the first feed-forward dense."""
    from ..interop.selivik import selivik
    layers = []
    for i in range(s["layers"]):
        if i % 4 == 0:
            entry = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
                     "softcap": 30.0, "mask": {"size": s["window"], "keep_first": s["keep"]}, "rot": {"base": 1e4, "dims": s["dim"], "scaling": {"factor": 4.0}}}}
        else:
            entry = {"type": "latent_attention", "mixer": {"heads": s["lat_heads"], "dim": s["lat_dim"], "rot_dim": s["rot"], "vdim": s["lat_vdim"], "kv_rank": s["rank"],
                     "q_rank": s["q_rank"], "scale": (s["lat_dim"] + s["rot"]) ** -0.5, "rot": {"base": 1e4, "dims": s["rot"]}}}
        entry["mlp"] = {"kind": "dense", "ff": s["dense"]} if i == 0 else \
            {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
        layers.append(entry)
    m = selivik(dtype=torch.bfloat16, device=device, vocab=s["vocab"], width=s["width"], norm={"eps": 1e-5}, embedding={"scale": s["width"] ** 0.5},
                residual_mult=0.5, layers=layers).eval()
    with torch.no_grad():
        for layer in m.layers:                                   # what bf16 releases hold
            if layer.sparse:
                layer.mlp.router.weight.copy_(layer.mlp.router.weight.to(torch.bfloat16).float())
    return m


def closest(s: dict, max_len: int, device="cuda"):
    from ..models.causal_transformer import CausalTransformer, Mixture, TransformerConfig
    # (its layers share one rotary table, as wide as the windowed layers' heads)
    return CausalTransformer(TransformerConfig(
        vocab_size=s["vocab"], emb_features=s["width"], num_layers=s["layers"], num_heads=s["heads"], num_kv_heads=s["kv"], head_dim=s["dim"], mlp_features=s["dense"],
        max_seq_len=max_len, norm_eps=1e-5, qk_norm=False, tie_embeddings=False, layer_types=("local", "mla", "mla", "mla"), window=s["window"],
        mixer_options=dict(kv_latent=s["rank"], q_latent=s["q_rank"], nope_dim=s["lat_dim"], rope_dim=s["rot"], v_dim=s["lat_vdim"]),
        mixture=Mixture(experts=s["experts"], top_k=s["top"], expert_features=s["ff"], layers=tuple(range(1, s["layers"])))), dtype=torch.bfloat16, device=device).eval()


@torch.no_grad()
def kernels(s: dict, tokens: int, decode_rows: int, context: int, iters: int) -> List[Dict[str, object]]:
    """Each kernel of the design and a like kernel: milliseconds and fraction of the roofline."""
    import torch.nn.functional as F

    from .. import ops
    from ..nn.kv_cache import CacheSlot, KVCache, KVStore, pool_width
    from ..ops import flash, latent, moe_serve, paged, rotary, streams
    from ..ops.routing import route
    pk = peaks()
    rand = lambda *sh: torch.randn(*sh, dtype=torch.bfloat16, device="cuda")
    d, H, G, D, C, keep = s["width"], s["heads"], s["kv"], s["dim"], s["window"], s["keep"]
    E, k, ff = s["experts"], s["top"], s["dense"]
    lat = latent.Latent(s["lat_heads"], s["lat_dim"], s["rot"], s["lat_vdim"], s["rank"], s["q_rank"], rotary.Rotary(s["rot"], 1e4, True))
    rows: List[Dict[str, object]] = []

    def entry(name, like, fn, nbytes, flops, fn2, nbytes2, flops2):
        line = {"kernel": name, "like": like}
        for tag, f, b, fl in (("", fn, nbytes, flops), ("like_", fn2, nbytes2, flops2)):
            ms = (replayed if name.startswith("decode") else timed)(f, iters)
            line[tag + "ms"] = ms
            line[tag + "of_roofline"] = max(b / pk["bytes"], fl / pk["flops"]) / ms * 1e3
        rows.append(line)

    T = tokens
    Hs, y, y2, w, x, br = torch.randn(T, 1, d, device="cuda"), rand(T, d), rand(T, d), rand(d), rand(T, d), rand(T, d)
    entry("stream_step (two sub-layers with scales, add, norm)", "stream_rms_norm", lambda: streams.stream_step(Hs, streams.Write(y, w, y2=y2, scale2=w, gain=0.5),
          None, w, 1e-5, torch.bfloat16, "rms", 1.0), T * d * 14, 0, lambda: ops.stream_rms_norm(x, br, w, 1e-5), T * d * 8, 0)
    del Hs, y, y2, br
    gu = rand(T, 2 * ff)
    entry("gelu_glu", "packed_swiglu", lambda: streams.gelu_glu(gu), T * ff * 6, 0, lambda: ops.packed_swiglu(gu), T * ff * 6, 0)
    del gu
    # windowed attention of prompts: the epilogue of the projection, the attention itself, a later portion
    S, R = 4096, max(1, T // 4096)
    heads, rot = paged.Heads(H, G, D, D), rotary.Rotary(D, 1e4, False, 4.0)
    slot = [CacheSlot(G, D, D)]
    store = KVStore(KVCache(page_size=64), 1, R, S, 0, 0, torch.bfloat16, "cuda", slots=slot)
    plain = KVStore(KVCache(page_size=64), 1, R, S, G, D, torch.bfloat16, "cuda")
    qkv, pos = rand(R, S, heads.row), torch.arange(S, device="cuda", dtype=torch.int32)[None].repeat(R, 1)
    bare = qkv.view(R, S, H + 2 * G, D)
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    bias, sinks = rand(heads.packed), torch.randn(H, device="cuda")
    cos, sin = ops.rope_tables(S, D, 1e4, "cuda")
    pos64, turned = pos.long(), paged.Turned(rot, rotary.angles(pos, rot))

    def rope_write():
        r = ops.rope(bare, cos, sin, pos64, rot_heads=H + G)
        plain.write(0, r[:, :, H:H + G], r[:, :, H + G:], pos64)
    nb = R * S * heads.packed * 2
    entry("head_norm_append with rotation", "rope + cache write", lambda: paged.qk_norm_append(qkv, heads, None, None, 1e-5, None, pos, pages, bias, turned, True),
          2 * nb + R * S * 2 * G * D * 2, 0, rope_write, 2 * nb + R * S * 2 * G * D * 2, 0)
    packed = paged.qk_norm_append(qkv, heads, None, None, 1e-5, None, pos, pages, bias, turned, True)
    q, kk, v = packed[:, :, :H], packed[:, :, H:H + G], packed[:, :, H + G:]
    seen = sum(min(i + 1, C) + min(keep, max(0, i + 1 - C)) for i in range(S)), sum(min(i + 1, C) for i in range(S))
    entry("flash, window with kept keys, soft cap and sinks", "flash, window", lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(C, 30.0, sinks,
          keep=keep)), 0, 4 * D * H * R * seen[0], lambda: flash.flash_fwd(q, kk, v, True, 0.1, False, flash.Variants(window=C)), 0, 4 * D * H * R * seen[1])
    at = S // 2
    q2, p2 = packed[:1, at:at + 512, :H].contiguous(), pos[:1, at:at + 512].contiguous()
    kc, vc = plain.gather(0, at + 512)
    entry(f"paged_attend_mma (512 after {at}, window)", "gathered score matrix", lambda: paged.paged_attend(q2, heads, p2, pages, 0.1, visible=paged.Visible(None,
          sinks, C, keep, 30.0)), 0, 4 * H * D * 512 * (C + keep), lambda: ops.attention_reference(q2, kc[:1], vc[:1], window=C), 0, 4 * H * D * 512 * C)
    del qkv, bare, packed, q, kk, v, store, plain, kc, vc, pages
    # latent attention of prompts
    W = pool_width(CacheSlot(1, lat.row, lat.rank, latent=True), torch.bfloat16)
    LH, dk, dv = lat.heads, lat.width, lat.vdim
    cols = lat.q_rank + lat.row + LH * dv
    store = KVStore(KVCache(page_size=64), 1, R, S, 0, 0, torch.bfloat16, "cuda", slots=[CacheSlot(1, lat.row, lat.rank, latent=True)])
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    z, qw, cw, up = rand(R, S, cols), rand(lat.q_rank), rand(lat.rank), rand(LH * (lat.dim + dv), lat.rank) * lat.rank ** -0.5
    table = rotary.angles(pos, lat.rotary)
    xn = rand(T, lat.q_rank + lat.row)
    wn = rand(lat.q_rank + lat.row)
    nb = R * S * (lat.q_rank + lat.row) * 4 + R * S * W * 2
    entry("latent_rows (norms, rotation, append)", "rms_norm", lambda: latent.rows(z, lat, qw, cw, 1e-5, table, pos, pages), nb, 0, lambda: ops.rms_norm(xn, wn, 1e-5),
          xn.numel() * 4, 0)
    q, gate = rand(R, S, LH, dk), z[..., lat.q_rank + lat.row:]
    c2, s2 = ops.rope_tables(S, lat.rot_dim, 1e4, "cuda")
    tail = rand(R, S, LH, lat.rot_dim)
    entry("rotate_tail", "rope", lambda: latent.rotate(q, lat, table), R * S * LH * lat.rot_dim * 4, 0, lambda: ops.rope(tail, c2, s2, pos64, rot_heads=LH),
          tail.numel() * 4, 0)
    _, made = latent.rows(z, lat, qw, cw, 1e-5, table, pos, pages)
    FD = 128 if dk > 64 else 64
    qf, kf, vf = rand(R, S, LH, FD), rand(R, S, LH, FD), rand(R, S, LH, FD)
    pairs = S * (S + 1) // 2
    up_flops = 2 * R * S * LH * (lat.dim + dv) * lat.rank
    entry("latent flash with gate, keys and values formed", f"flash, heads of {FD}", lambda: latent.flash(q, made, up, lat, 0.1, gate), 0,
          2 * (dk + dv) * LH * R * pairs + up_flops, lambda: flash.flash_fwd(qf, kf, vf, True, 0.1, False), 0, 4 * FD * LH * R * pairs)
    entry("up-projection alone (vendor)", "the same", lambda: ops.linear(made.c, up), 0, up_flops, lambda: ops.linear(made.c, up), 0, up_flops)
    del qf, kf, vf
    from ..nn.mla import MultiHeadLatentAttention
    old = MultiHeadLatentAttention(d, LH, lat.rank, lat.q_rank, lat.dim, lat.rot_dim, dv, dtype=torch.bfloat16, device="cuda")
    q2, p2 = q[:1, at:at + 512].contiguous(), pos[:1, at:at + 512].contiguous()
    lens = torch.full((1,), at + 512, dtype=torch.int32, device="cuda")
    one = pages._replace(table=pages.table[:1])
    rowsd = torch.cat([made.c[:1, :at + 512], made.key[:1, :at + 512]], -1)
    fl = 2 * (dk + dv) * LH * sum(at + i + 1 for i in range(512)) + 2 * (at + 512) * LH * (lat.dim + dv) * lat.rank
    entry(f"latent portion (512 after {at}: gather, keys and values formed, flash)", "latent scores in PyTorch",
          lambda: latent.flash(q2, latent.gather(lat, lens, at + 512, one), up, lat, 0.1), 0, fl,
          lambda: old._absorbed(q2[..., :lat.dim], q2[..., lat.dim:], rowsd, p2.long(), lens), 0, fl)
    del z, q, made, store, pages, tail, xn, old
    torch.cuda.empty_cache()
    # a decode step
    B = decode_rows
    store = KVStore(KVCache(page_size=64), 1, B, context + 64, 0, 0, torch.bfloat16, "cuda", slots=[CacheSlot(1, lat.row, lat.rank, latent=True)])
    plain = KVStore(KVCache(page_size=64), 1, B, context + 64, G, D, torch.bfloat16, "cuda")
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    q1, posd = rand(B, 1, LH, dk), torch.full((B, 1), context, device="cuda", dtype=torch.int32)
    lens = torch.full((B,), context + 1, device="cuda")
    t1 = rotary.angles(posd, lat.rotary)
    qa = latent.absorb(q1, up, lat, t1, W)
    lend = lambda n, width: store._partials(n, width, "cuda")
    q0 = rand(B, H, D)
    nb, nb2 = B * (context + 1) * lat.row * 2, B * (context + 1) * 2 * G * D * 2
    entry("decode: latent_attend", "decode attention", lambda: latent.attend(qa, lat, posd, pages, 0.1, store.max_len, lend), nb,
          2 * (lat.row + lat.rank) * LH * B * (context + 1), lambda: plain.decode_attention(0, q0, lens), nb2, 0)
    wk, wv = lat.split_up(up)
    wk, wv, qh = wk.contiguous(), wv.transpose(1, 2).contiguous(), q1[:, 0, :, :lat.dim].transpose(0, 1).contiguous()
    entry("decode: head_product (queries, rotation)", "batched vendor product", lambda: latent.absorb(q1, up, lat, t1, W), wk.numel() * 2 + q1.numel() * 2 + qa.numel() * 2,
          0, lambda: torch.bmm(qh, wk), wk.numel() * 2 + q1.numel() * 2 + qa.numel() * 2, 0)
    o = latent.attend(qa, lat, posd, pages, 0.1, store.max_len, lend)
    oh, g1 = o[:, 0].transpose(0, 1).contiguous(), rand(B, 1, LH * dv)
    entry("decode: head_product (values, gate)", "batched vendor product", lambda: latent.expand(o, up, lat, g1), wv.numel() * 2 + o.numel() * 2 + B * LH * dv * 4, 0,
          lambda: torch.bmm(oh, wv), wv.numel() * 2 + o.numel() * 2 + B * LH * dv * 2, 0)
    del store, pages
    store = KVStore(KVCache(page_size=64), 1, B, context + 64, 0, 0, torch.bfloat16, "cuda", slots=slot)
    qkv1 = rand(B, 1, heads.row)
    entry("decode: windowed attention (norms, rotation, append, paged)", "decode attention, window", lambda: store.attend_slot(0, qkv1, heads, posd, scale=0.1,
          eps=1e-5, bias=bias, sinks=sinks, window=C, keep=keep, softcap=30.0, rot=rot, unit=True), B * min(C + keep, context + 1) * 2 * G * D * 2, 0,
          lambda: plain.decode_attention(0, q0, lens, window=C), B * min(C, context + 1) * 2 * G * D * 2, 0)
    del store, plain
    # the router
    sel = moe_serve.Selection(E, k, score="top_softmax")
    wr, b = torch.randn(E, d, device="cuda").to(torch.bfloat16).float() * d ** -0.5, torch.randn(E, device="cuda") * 0.1
    split = moe_serve.split_weights(wr)
    for tag, n in (("prompt", T), ("decode", decode_rows)):
        xs = x[:n].contiguous()
        entry("router" if tag == "prompt" else "decode: router", "fp32 router product + moe_route", lambda: moe_serve.route(xs, wr, split, None, sel, logit_bias=b), n * d * 2 + E * d * 2, 2 * n * E * d,
              lambda: route(F.linear(xs.float(), wr), None, k, "softmax", True), n * d * 2 + E * d * 4, 2 * n * E * d)
    return rows
