"""Prefill and decode throughput of a decoder design beside this library's closest decoder of the same sizes, and each of the design's kernels
beside the like kernel of that decoder, as a fraction of its roofline: the Ragenex design here (closest: rotary attention and gated-delta-net
layers in the same order, SwiGLU, one bf16 residual), the Fakonex design in ``telemetry.fakonex_bench``, the Selivik design in
``telemetry.selivik_bench``, the Rarelorn design in ``telemetry.rarelorn_bench``.

``bench.py --decoder ragenex | fakonex | selivik | rarelorn`` prints the result as one JSON line.  Weights are random.  Everything is timed on the device with CUDA events
after warm-up; prefill activations and weights are larger than L2, and a decode step (one CUDA graph, where the model's step can be captured) streams
all the weights.
"""
from __future__ import annotations

import json
from pathlib import Path
from typing import Callable, Dict, List, Optional

import torch

WARMUP = 3
SIZES = {
    "d2048": dict(width=2048, heads=16, kv=4, dim=128, ff=5632, lin=16, lin_dim=128, layers=8, vocab=32768),
    "d4096": dict(width=4096, heads=32, kv=8, dim=128, ff=14336, lin=32, lin_dim=128, layers=8, vocab=32768),
    "d2048h64": dict(width=2048, heads=32, kv=8, dim=64, ff=5632, lin=16, lin_dim=128, layers=8, vocab=32768),
}
STREAMS = 2


def peaks() -> Dict[str, float]:
    """Measured copy bandwidth and cuBLAS bf16 rate where the checkout has them, else this pool's earlier figures."""
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        m = json.loads(f.read_text())
        return {"bytes": m["hbm_gbs"] * 1e9, "flops": m["bf16_tflops"] * 1e12, "source": "measured"}
    return {"bytes": 6.65e12, "flops": 1.59e15, "source": "fallback"}


def timed(fn: Callable[[], object], iters: int) -> float:
    """Milliseconds per call."""
    for _ in range(WARMUP):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def replayed(fn: Callable[[], object], iters: int, copies: int = 8) -> float:
    """Milliseconds per call inside a CUDA graph of ``copies`` calls (kernels of a decode step, which launches from Python would hide)."""
    fn()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for _ in range(copies):
            fn()
    return timed(graph.replay, iters) / copies


def ragenex(s: dict, max_len: int, device="cuda"):
    """The design at size ``s``: every fourth layer lightning attention."""
    from ..models.causal_transformer import CausalTransformer, TransformerConfig
    n = s["layers"]
    kinds = tuple("lightning" if i % 4 == 3 else "nope" for i in range(n))
    decay = [1 - 2.0 ** -(2 + 6 * h / s["lin"]) for h in range(s["lin"])]
    options = tuple({"num_heads": s["lin"], "head_dim": s["lin_dim"], "decay": decay} if k == "lightning" else {} for k in kinds)
    return CausalTransformer(TransformerConfig(
        vocab_size=s["vocab"], emb_features=s["width"], num_layers=n, num_heads=s["heads"], num_kv_heads=s["kv"], head_dim=s["dim"],
        mlp_features=s["ff"], max_seq_len=max_len, norm_eps=1e-5, qk_norm=False, qk_norm_full=True, tie_embeddings=False, norm="layer",
        layer_types=kinds, layer_options=options, mlp_activation="clamped_glu", query_temperature=(0.1, 1024), query_scale=s["dim"] ** -0.5,
        hyper_connections=STREAMS, hyper_dynamic=False, layer_scale=True, learned_positions=True), dtype=torch.bfloat16, device=device).eval()


def closest(s: dict, max_len: int, device="cuda"):
    from ..models.causal_transformer import CausalTransformer, TransformerConfig
    kinds = tuple("gdn" if i % 4 == 3 else "attention" for i in range(s["layers"]))
    return CausalTransformer(TransformerConfig(
        vocab_size=s["vocab"], emb_features=s["width"], num_layers=s["layers"], num_heads=s["heads"], num_kv_heads=s["kv"], head_dim=s["dim"],
        mlp_features=s["ff"], max_seq_len=max_len, norm_eps=1e-5, qk_norm=False, tie_embeddings=False, layer_types=kinds,
        mixer_options=dict(num_k_heads=s["lin"], num_v_heads=s["lin"], head_k_dim=s["lin_dim"], head_v_dim=s["lin_dim"])),
        dtype=torch.bfloat16, device=device).eval()


def keeps_latents(model) -> bool:
    """Whether some layer keeps its latents outside the pages (``KVStore.latent``): its cached step forms a prompt's score matrix and reads lengths on the
    host, so a prompt is timed as a whole sequence without a cache and a decode step without a graph."""
    return any(k == "mla" and layer.mixer.shape is None for k, layer in zip(model.config.kinds(), model.layers))


@torch.no_grad()
def throughput(model, s: dict, rows: int, prompt: int, decode_rows: int, context: int, iters: int) -> Dict[str, float]:
    from ..nn.kv_cache import KVCache
    from ..nn.linear_attention import RecurrentCache
    from ..sampling.text import make_cache
    for p in model.parameters():
        p.requires_grad_(False)
    g = torch.Generator(device="cuda").manual_seed(0)

    def cache(n, length):
        store = make_cache(model, n, length, KVCache(page_size=64))
        return store, (store if store.slots is not None else RecurrentCache(store))

    ids = torch.randint(0, s["vocab"], (rows, prompt), device="cuda", generator=g)
    pos = torch.arange(prompt, device="cuda")[None].repeat(rows, 1)
    store, c = cache(rows, prompt)
    store.chunk_span = (0, prompt)
    uncached = keeps_latents(model)

    def prefill():
        if uncached:
            return model.logits(model(ids, return_hidden=True)[:, -1])
        return model.logits(model(ids, positions=pos, cache=c, return_hidden=True)[:, -1])
    ms = timed(prefill, iters)
    out = {"prefill_tokens_per_s": rows * prompt / ms * 1e3, "prefill_ms": ms}
    del store, c
    store, c = cache(decode_rows, context + 64)
    tok = torch.randint(0, s["vocab"], (decode_rows, 1), device="cuda", generator=g)
    at = torch.full((decode_rows, 1), context, device="cuda")

    def step():
        return model.next_tokens_greedy(model(tok, positions=at, cache=c, return_hidden=True)[:, 0])
    if uncached:
        ms = timed(step, 2 * iters)
        out.update(decode_tokens_per_s=decode_rows / ms * 1e3, decode_ms=ms, eager=True)
        del store, c
        torch.cuda.empty_cache()
        return out
    side = torch.cuda.Stream()
    torch.cuda.synchronize()                      # (the inputs above are made on the other stream)
    with torch.cuda.stream(side):
        step()
        step()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        step()
    ms = timed(graph.replay, 10 * iters)
    out.update(decode_tokens_per_s=decode_rows / ms * 1e3, decode_ms=ms)
    del graph, store, c
    torch.cuda.empty_cache()
    return out


@torch.no_grad()
def kernels(s: dict, tokens: int, decode_rows: int, context: int, iters: int) -> List[Dict[str, object]]:
    """Each kernel of the design and the like kernel of the closest model: milliseconds and fraction of the roofline."""
    from .. import ops
    from ..nn.kv_cache import CacheSlot, KVCache, KVStore
    from ..ops import decayed, gdn, paged, streams
    pk = peaks()
    bf = dict(dtype=torch.bfloat16, device="cuda")
    rand = lambda *sh: torch.randn(*sh, **bf)
    d, F, H, G, D, L, W = s["width"], s["ff"], s["heads"], s["kv"], s["dim"], s["lin"], s["lin_dim"]
    rows: List[Dict[str, object]] = []

    def entry(name, like, fn, nbytes, flops, fn2, nbytes2, flops2):
        line = {"kernel": name, "like": like}
        for tag, f, b, fl in (("", fn, nbytes, flops), ("like_", fn2, nbytes2, flops2)):
            ms = timed(f, iters)
            line[tag + "ms"] = ms
            line[tag + "of_roofline"] = max(b / pk["bytes"], fl / pk["flops"]) / ms * 1e3
        rows.append(line)

    T, n = tokens, STREAMS
    Hs, y, w = torch.randn(T, n, d, device="cuda"), rand(T, d), rand(d)
    write = streams.Write(y, w, torch.eye(n, device="cuda") * 0.5, torch.full((n,), 0.1, device="cuda"))
    read = torch.full((n,), 0.5, device="cuda")
    x, br = rand(T, d), rand(T, d)
    entry("stream_step", "stream_rms_norm", lambda: streams.stream_step(Hs, write, read, w, 1e-5, torch.bfloat16), T * d * (8 * n + 4), 0,
          lambda: ops.stream_rms_norm(x, br, w, 1e-5), T * d * 8, 0)
    del Hs, y, x, br
    gu = rand(T, 2 * F)
    entry("clamped_glu", "packed_swiglu", lambda: streams.clamped_glu(gu, 7.0), T * F * 6, 0, lambda: ops.packed_swiglu(gu), T * F * 6, 0)
    del gu
    # projection epilogue of a prompt; the closest model rotates in place and writes the cache from the packed projection
    S, R = 4096, max(1, T // 4096)
    store = KVStore(KVCache(page_size=64), 1, R, S, 0, 0, torch.bfloat16, "cuda", slots=[CacheSlot(G, D, D)])
    heads = paged.Heads(H, G, D, D)
    qkv, pos = rand(R, S, heads.packed), torch.arange(S, device="cuda", dtype=torch.int32)[None].repeat(R, 1)
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    qw, kw = rand(H * D), rand(G * D)
    plain = KVStore(KVCache(page_size=64), 1, R, S, G, D, torch.bfloat16, "cuda")
    cos, sin = ops.rope_tables(S, D, 1e4, "cuda")
    pos64 = pos.long()

    def rope_write():
        r = ops.rope(qkv.view(R, S, H + 2 * G, D), cos, sin, pos64, rot_heads=H + G)
        plain.write(0, r[:, :, H:H + G], r[:, :, H + G:], pos64)
    nb = R * S * heads.packed * 2
    entry("qk_norm_append", "rope + cache write", lambda: paged.qk_norm_append(qkv, heads, qw, kw, 1e-5, (0.1, 1024), pos, pages),
          2 * nb + R * S * 2 * G * D * 2, 0, rope_write, 2 * nb + R * S * 2 * G * D * 2, 0)
    # a prompt's later portion against what the cache holds (the closest model gathers the pages and forms the score matrix)
    half = S // 2
    packed = paged.qk_norm_append(qkv, heads, qw, kw, 1e-5, None, pos, pages)
    q2, p2 = packed[:1, half:half + 512, :H].contiguous(), pos[:1, half:half + 512].contiguous()
    fl = 4 * H * D * 512 * (half + 256)
    kc, vc = plain.gather(0, half + 512)
    entry("paged_attend_mma (512 after 2048)", "gathered score matrix", lambda: paged.paged_attend(q2, heads, p2, pages, 0.1), 0, fl,
          lambda: ops.attention_reference(q2, kc[:1], vc[:1]), 0, fl)
    del qkv, packed, store, plain, kc, vc, pages
    # the recurrence over a prompt
    x = rand(R, S, 3 * L * W)
    decay = torch.linspace(0.9, 0.999, L, device="cuda")
    state = torch.zeros(R, L, W, W, device="cuda")
    q, k, v = (t.contiguous() for t in torch.nn.functional.normalize(x.view(R, S, 3, L, W), dim=-1).unbind(2))
    gg, beta = -torch.rand(R, S, L, device="cuda") * 0.1, torch.rand(R, S, L, device="cuda")
    per = R * S * L
    entry("decayed_chunks", "gated delta rule (gdn_sm100)", lambda: decayed.decayed_attention(x, decay, L, W, W, state, pos),
          per * W * 8, per * (64 * 2 * W + 4 * W * W),
          lambda: gdn.gated_delta_rule(q, k, v, gg, beta, None, None), per * (W * 8 + 8), per * (64 * 4 * W + 64 * 2 * W + 6 * W * W))
    del x, q, k, v, gg, beta
    o, gate, nw = rand(T, L * W), rand(T, L * W), rand(L * W)
    entry("sigmoid_gated_norm", "gated_rms_norm", lambda: streams.sigmoid_gated_norm(o, gate, nw, 1e-5), T * L * W * 6, 0,
          lambda: ops.gated_rms_norm(o, gate, nw, 1e-5), T * L * W * 6, 0)
    del o, gate
    # decode: the state of many rows against the keys and values of as many rows
    B = decode_rows
    x1, st, p1 = rand(B, 1, 3 * L * W), torch.zeros(B, L, W, W, device="cuda"), torch.full((B, 1), context, device="cuda", dtype=torch.int32)
    q1, k1, v1 = (t.contiguous() for t in x1.view(B, 3, L, W).unbind(1))
    g1, b1, st2 = -torch.rand(B, L, device="cuda"), torch.rand(B, L, device="cuda"), st.clone()
    from ..ops.scan import gated_delta_rule_step
    entry("decayed_step", "gated_delta_rule_step", lambda: decayed.decayed_attention(x1, decay, L, W, W, st, p1), B * L * W * W * 8, 0,
          lambda: gated_delta_rule_step(q1, k1, v1, g1, b1, st2), B * L * W * W * 8, 0)
    del st, st2
    store = KVStore(KVCache(page_size=64), 1, B, context + 64, 0, 0, torch.bfloat16, "cuda", slots=[CacheSlot(G, D, D)])
    plain = KVStore(KVCache(page_size=64), 1, B, context + 64, G, D, torch.bfloat16, "cuda")
    q1, lens, posd = rand(B, 1, heads.packed), torch.full((B,), context + 1, device="cuda"), torch.full((B, 1), context, device="cuda")
    nb = B * (context + 1) * 2 * G * D * 2
    entry("decode attention (norm, append, paged)", "decode attention", lambda: store.attend_slot(0, q1, heads, posd, scale=0.1, eps=1e-5, q_weight=qw,
          k_weight=kw, temperature=(0.1, 1024)), nb, 0, lambda: plain.decode_attention(0, q1.view(B, H + 2 * G, D)[:, :H], lens), nb, 0)
    return rows


def run(name: str = "ragenex", sizes=None, rows: int = 4, prompt: int = 4096, decode_rows: int = 64, context: Optional[int] = None, iters: int = 5) -> Dict[str, object]:
    torch.manual_seed(0)
    if name == "fakonex":
        from . import fakonex_bench as f
        table, design, near, parts = f.SIZES, f.design, f.closest, f.kernels
        context = 4095 if context is None else context           # the last position of a chunk: as many keys as the closest model's window holds
    elif name in ("selivik", "rarelorn"):
        if name == "selivik":
            from . import selivik_bench as f
        else:
            from . import rarelorn_bench as f
        table, design, near, parts = f.SIZES, f.design, f.closest, f.kernels
        context = 4096 if context is None else context
    else:
        table, design, near, parts = SIZES, ragenex, closest, kernels
        context = 4096 if context is None else context
    out: Dict[str, object] = {"peaks": peaks(), "rows": rows, "prompt": prompt, "decode_rows": decode_rows, "context": context, "warmup": WARMUP,
                              "dtype": "bf16", "data": "synthetic (random token ids, random-init weights)", "sizes": {}}
    for size in sizes or table:
        s = table[size]
        line: Dict[str, object] = {"config": s}
        for tag, make in ((name, design), ("closest", near)):
            line[tag] = throughput(make(s, prompt + 128), s, rows, prompt, decode_rows, context, iters)
            torch.cuda.empty_cache()
        line["kernels"] = parts(s, rows * prompt, decode_rows, context, iters)
        torch.cuda.empty_cache()
        out["sizes"][size] = line
    return out
