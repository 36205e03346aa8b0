"""The Fakonex design on a GPU: its kernels against the plain PyTorch forms, whole models in fp32 and bf16 against the restated decoder on
every schedule, and generation through both entry points (the server with its CUDA graph)."""
import pytest
import torch

import fakonex_cases as C
import fakonex_oracle as O

from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore
from dew_b200.ops import moe_serve, paged, streams

pytestmark = pytest.mark.gpu
DEV = "cuda"


def rnd(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype).to(DEV)


def close(got, want, rel):
    return got.shape == want.shape and float((got.float() - want.float()).abs().max()) <= rel * float(want.float().abs().max().clamp_min(1e-6))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d", [(1, 64), (1, 4096), (1, 1100), (1, 7), (3, 260), (5, 33)])
def test_residual_step_with_a_norm_on_what_joins(dtype, n, d):
    rel = 1e-5 if dtype == torch.float32 else 1e-2
    T = 9
    H, y, wy, w = rnd(T, n, d, seed=2), 5 * rnd(T, d, seed=3, dtype=dtype), rnd(d, seed=4, dtype=dtype), rnd(d, seed=5, dtype=dtype)
    mix, out = rnd(n, n, seed=6), rnd(n, seed=7)
    for norm in ("rms", "layer"):
        for write in (streams.Write(y, weight=wy, eps=0.1), streams.Write(y, None, mix, out, wy, 0.1), streams.Write(y, w), streams.Write(y)):
            ref, H_ref = streams.stream_step_reference(H, write, None, w, 1e-2, dtype, norm)
            got, H_got = streams.stream_step(H.clone(), write, None, w, 1e-2, dtype, norm)
            assert close(H_got, H_ref, 1e-5) and close(got, ref, rel)
    _, H_got = streams.stream_step(H.clone(), streams.Write(y, weight=wy, eps=0.1), None, None, 0.0, dtype)
    assert close(H_got, streams.stream_step_reference(H, streams.Write(y, weight=wy, eps=0.1), None, None, 0.0, dtype)[1], 1e-5)
    x = 9 * rnd(T, d, seed=8, dtype=dtype)
    assert close(streams.softcap(x, 4.0), streams.softcap_reference(x, 4.0), 1e-6)


HEADS = [paged.Heads(5, 1, 96, 88, True, True), paged.Heads(8, 2, 64, 64, True, True), paged.Heads(6, 2, 128, 80, True, True),
         paged.Heads(12, 1, 24, 40, True, False), paged.Heads(2, 2, 200, 130, True, True), paged.Heads(3, 1, 7, 5, True, True)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads", HEADS)
def test_projection_epilogue_and_head_gate(dtype, heads):
    rel = 1e-5 if dtype == torch.float32 else 1e-2
    H, G, dk, dv = heads
    D = max(8, (max(dk, dv) + 7) // 8 * 8)
    for h in (heads, paged.Heads(H, G, dk, dv, False, heads.gated)):
        qkv, bias, qw, kw = rnd(2, 37, h.row, dtype=dtype), rnd(h.packed, seed=1, dtype=dtype), rnd(dk, seed=2, dtype=dtype), rnd(dk, seed=3, dtype=dtype)
        pos = torch.stack([torch.arange(37), torch.cat([torch.arange(5, 25), torch.full((17,), -1)])]).to(torch.int32)
        pools = [torch.zeros(9, 16, G, D, dtype=dtype, device=DEV) for _ in range(2)]
        table = torch.tensor([[3, 1, 7], [2, 8, 4]], dtype=torch.int32)
        got = paged.qk_norm_append(qkv, h, qw, kw if h.own else None, 1e-2, None, pos.to(DEV), paged.Pages(*pools, table.to(DEV), 16, None), bias)
        cpu = [p.cpu().float().zero_() for p in pools]
        want = paged.qk_norm_append(qkv.cpu().float(), h, qw.cpu().float(), kw.cpu().float() if h.own else None, 1e-2, None, pos,
                                    paged.Pages(*cpu, table, 16, None), bias.cpu().float())
        assert close(got.cpu(), want, rel)
        assert all(close(a.cpu(), b, rel) for a, b in zip(pools, cpu))
        if h.gated:
            o = got[:, :, :H].contiguous()
            assert close(paged.head_gate(o, qkv[..., h.packed:], dv), paged.head_gate_reference(o, qkv[..., h.packed:], dv), rel)


@pytest.mark.parametrize("S,D,Hq,Hkv,chunk", [(512, 128, 4, 2, 96), (512, 128, 4, 1, 128), (640, 64, 2, 2, 300), (384, 64, 3, 1, 1), (256, 128, 2, 1, 1000),
                                             (1280, 128, 2, 1, 512)])
def test_flash_forward_in_chunks(S, D, Hq, Hkv, chunk):
    from dew_b200.ops.flash import Variants, flash_fwd
    from dew_b200.ops.functional import attention_reference
    q, k, v = (rnd(2, S, h, D, seed=i, dtype=torch.bfloat16) for i, h in enumerate((Hq, Hkv, Hkv)))
    q = q * 2
    sinks = rnd(Hq, seed=5) + 1
    seg = (torch.arange(S, device=DEV, dtype=torch.int32) // chunk + 1)[None].expand(2, S)
    for s in (None, sinks):
        got, lse = flash_fwd(q, k, v, True, 0.1, var=Variants(chunk=chunk, sinks=s))
        want = attention_reference(q.float(), k.float(), v.float(), True, 0.1, sinks=s, segment_ids=seg)
        assert close(got, want, 1.5e-2) and bool(torch.isfinite(lse).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [1, 48, 64, 100, 128, 257, None])
@pytest.mark.parametrize("heads", HEADS)
def test_attention_from_the_packed_projection(dtype, heads, chunk):
    """``attend_slot`` and a layer that shares the slot's keys: a prompt, portions at mixed positions, and decode steps past chunk borders, with
    planted keys just inside and just outside chunks and at page borders."""
    rel = 2e-5 if dtype == torch.float32 else 6e-2      # bf16 queries and keys under sharp scores; a missed key is past 0.2
    H, G, dk, dv = heads
    other = paged.Heads(H, G, dk, dv, False, heads.gated)
    rows, first, T = 3, 128, 300
    kw = dict(scale=dk ** -0.5, eps=1e-3, q_weight=2 * rnd(dk, seed=1, dtype=dtype).abs() + 0.5, k_weight=rnd(dk, seed=2, dtype=dtype),
              bias=0.3 * rnd(heads.packed, seed=4, dtype=dtype), sinks=rnd(H, seed=5, dtype=dtype), chunk=chunk)
    slots = [CacheSlot(G, dk, dv), CacheSlot(G, dk, dv, source=0)]
    store = KVStore(KVCache(page_size=64, pages=24), 2, rows, 320, 0, 0, dtype, DEV, slots=slots)
    store.page_table.copy_(torch.randperm(24, generator=torch.Generator().manual_seed(0))[:15].reshape(3, 5).to(DEV))
    cpu = KVStore(KVCache(page_size=64, pages=24), 2, rows, 320, 0, 0, torch.float32, "cpu", slots=slots)
    cpu.page_table.copy_(store.page_table.cpu())
    ckw = {k: v.float().cpu() if isinstance(v, torch.Tensor) else v for k, v in kw.items()}
    x = rnd(rows, T, heads.row, seed=3, dtype=dtype)
    k = x[..., H * dk:(H + G) * dk] + kw["bias"][H * dk:(H + G) * dk]
    for at in range(130, T, 13):                                       # queries that point at one key: around the chunk's start, and page borders
        lo = at // chunk * chunk if chunk else 0
        for r, target in enumerate((lo, max(lo - 1, 0), min(at, (at // 64) * 64))):
            q = k[r, target].view(G, dk).repeat_interleave(H // G, 0) * kw["k_weight"] / kw["q_weight"]
            x[r, at, :H * dk] = 4 * q.reshape(-1) - kw["bias"][:H * dk]
    skw = lambda d: {**d, "k_weight": None, "bias": d["bias"][:H * dk], "chunk": None if chunk is None else chunk + 13}

    def both(b, starts):
        n = max(e - s for s, e in zip(starts, b))
        xs, pos = torch.zeros(rows, n, heads.row, dtype=dtype, device=DEV), torch.full((rows, n), -1)
        for r in range(rows):
            xs[r, :b[r] - starts[r]] = x[r, starts[r]:b[r]]
            pos[r, :b[r] - starts[r]] = torch.arange(starts[r], b[r])
        dpos = pos.to(DEV)
        for slot, h, kwargs, cargs in ((0, heads, kw, ckw), (1, other, skw(kw), skw(ckw))):
            part = xs if slot == 0 else torch.cat([xs[..., :H * dk], xs[..., heads.packed:]], -1)
            got = store.attend_slot(slot, part, h, dpos, **kwargs)
            want = cpu.attend_slot(slot, part.float().cpu(), h, pos, **cargs)
            for r in range(rows):
                m = b[r] - starts[r]
                assert m == 0 or close(got[r, :m].cpu(), want[r, :m], rel), (slot, starts, b, r)
                assert bool(torch.isfinite(got[r]).all())

    at = [first, 77, 1]
    both(at, [0, 0, 0])
    for nxt in ([first + 2, 77 + 61, 1], [199, 199, 130]):
        both(nxt, at)
        at = nxt
    for t in range(101):
        nxt = [min(at[0] + 1, T), at[1] + (t % 3 > 0), at[2] + 1]
        both(nxt, at)
        at = nxt


@pytest.mark.parametrize("heads", [h for h in HEADS if max(h.dk, h.dv) <= 256])
@pytest.mark.parametrize("chunk", [None, 1, 50, 64])
def test_tensor_core_and_general_paged_attention_agree(heads, chunk):
    H, G, dk, dv = heads
    D = next(d for d in (64, 128, 256) if d >= max(dk, dv))
    pages = paged.Pages(rnd(9, 64, G, D, seed=1, dtype=torch.bfloat16), rnd(9, 64, G, D, seed=2, dtype=torch.bfloat16),
                        torch.tensor([[3, 1, 7, 0], [2, 8, 4, 5]], dtype=torch.int32, device=DEV), 64, torch.tensor([1, 0], dtype=torch.int32, device=DEV))
    for t in (pages.k, pages.v):
        t[..., dk if t is pages.k else dv:] = 0
    pos = torch.stack([torch.arange(100, 170), torch.cat([torch.arange(5, 60), torch.full((15,), -1)])]).to(torch.int32).to(DEV)
    q = rnd(2, 70, H, D, seed=3, dtype=torch.bfloat16)
    q[..., dk:] = 0
    gate, visible = rnd(2, 70, H + 3, seed=4, dtype=torch.bfloat16)[..., 3:], paged.Visible(chunk, rnd(H, seed=5))
    a, b = (paged.paged_attend(q, heads, pos, pages, 0.2, kernel=k, visible=visible, gate=gate) for k in ("mma", "general"))
    ref = paged.head_gate_reference(paged.paged_attend_reference(q.float(), heads, pos, pages._replace(k=pages.k.float(), v=pages.v.float()), 0.2, visible),
                                    gate.float(), dv)
    assert close(a, ref, 1e-2) and close(b, ref, 1e-2) and bool((a[1, 55:] == 0).all())


@pytest.mark.parametrize("D,Hq,Hkv", [(128, 8, 2), (128, 16, 1), (64, 8, 2)])
def test_decode_in_chunks_over_long_rows(D, Hq, Hkv):
    """Rows at and around chunk borders, with chunks of many tiles (the balanced kernel cuts them into parts) and off the page grid."""
    heads = paged.Heads(Hq, Hkv, D, D)
    lens = [1, 64, 1000, 1001, 2000, 2001, 2999, 4000, 4064]
    store = KVStore(KVCache(page_size=64), 1, len(lens), 4096, 0, 0, torch.bfloat16, DEV, slots=[CacheSlot(Hkv, D, D)])
    store.k[0].copy_(rnd(*store.k[0].shape, seed=1)), store.v[0].copy_(rnd(*store.v[0].shape, seed=2))
    for chunk in (1000, 512, 96, None):
        qkv, pos = rnd(len(lens), 1, heads.packed, seed=3, dtype=torch.bfloat16), torch.tensor(lens, device=DEV)[:, None] - 1
        sinks = rnd(Hq, seed=6)
        got = store.attend_slot(0, qkv, heads, pos, scale=0.2, chunk=chunk, sinks=sinks)
        pages = paged.Pages(store.k[0].float(), store.v[0].float(), store.page_table, 64, None)
        want = paged.paged_attend_reference(qkv[..., :Hq * D].view(len(lens), 1, Hq, D).float(), heads, pos.int(), pages, 0.2, paged.Visible(chunk, sinks))
        assert close(got, want, 1.5e-2), chunk


# ------------------------------------------------------------------------------------------------ experts
SELECTIONS = [moe_serve.Selection(10, 3, 2, 1, float("-inf"), "sigmoid"), moe_serve.Selection(12, 2, 4, 2, float("-inf"), "sigmoid", True, 2.5),
              moe_serve.Selection(5, 5, 1, 1, 0.0, "softmax", False), moe_serve.Selection(128, 8, 8, 4, 0.0, "sigmoid"),
              moe_serve.Selection(300, 20, 10, 3, float("-inf"), "softmax"), moe_serve.Selection(6, 3, 6, 4, float("-inf"), "sigmoid")]


def mixture_reference(x, ids, w, gate_up, down, shared, gate_w):
    y = torch.zeros(x.shape[0], down.shape[1], dtype=torch.float64)
    for t in range(x.shape[0]):
        for e, a in zip(ids[t].tolist(), w[t].tolist()):
            if e >= 0:
                g, u = (gate_up[e] @ x[t]).chunk(2)
                y[t] += a * (down[e] @ (O.silu(g) * u))
        if shared is not None:
            y[t] += (1.0 if gate_w is None else O.sigmoid(gate_w @ x[t])) * shared[t]
    return y


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d,F,s", [(1, 64, 24, SELECTIONS[0]), (37, 72, 40, SELECTIONS[1]), (70, 30, 7, SELECTIONS[2]), (90, 128, 16, SELECTIONS[3]),
                                     (40, 64, 8, SELECTIONS[4]), (700, 48, 32, SELECTIONS[5]), (600, 64, 64, SELECTIONS[3])])
def test_served_experts(dtype, T, d, F, s):
    """Selection (both forms of the router, weights that bf16 holds and that it does not), sorted rows, grouped products and the weighted sum."""
    E = s.experts
    x, b = rnd(T, d, dtype=dtype), rnd(E, seed=1) * 0.3 - 1.0
    gate_up, down = 2 * d ** -0.5 * rnd(E, 2 * F, d, seed=3), F ** -0.5 * rnd(E, d, F, seed=4)
    gate_up, down, gw = gate_up.to(dtype), down.to(dtype), rnd(1, d, seed=5, dtype=dtype) * d ** -0.5
    shared = rnd(T, d, seed=6, dtype=dtype)
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    pos[T // 2:T // 2 + max(T // 8, 0)] = -1
    live = (pos >= 0).cpu()
    for exact in (True, False):
        weight = 2 * d ** -0.5 * rnd(E, d, seed=2)
        weight = weight.to(torch.bfloat16).float() if exact else weight
        split = moe_serve.split_weights(weight)
        assert split.exact == exact
        logits = x.double() @ weight.double().t()
        scores = torch.softmax(logits, -1) if s.score == "softmax" else torch.sigmoid(logits)
        choice = moe_serve.choice_scores(scores.cpu(), b.double().cpu(), s)
        for form in ["rows"] + (["product"] if dtype == torch.bfloat16 and d % 8 == 0 else []):
            r = moe_serve.route(x, weight, split if dtype == torch.bfloat16 else None, b, s, pos, kernel=form)
            ids = r.ids.cpu().long()
            assert bool((ids[~live] == -1).all()) and int(r.counts.sum()) == int(live.sum()) * s.top
            top = choice.topk(s.top, -1).values[:, -1]
            # what was chosen is within rounding of the best, nothing twice, nothing from a dropped group
            assert bool((choice.gather(1, ids.clamp_min(0))[live] >= top[live, None] - 2e-5).all())
            assert all(len(set(row)) == s.top for row in ids[live].tolist())
            want = scores.cpu().gather(1, ids.clamp_min(0))
            want = (want / (want.sum(-1, keepdim=True) + 1e-20) if s.norm else want) * s.scaling
            assert close(r.weights.cpu()[live].double(), want[live], 1e-5)
            assert bool((torch.bincount(ids[live].flatten(), minlength=E) == r.counts.cpu()).all())
    got = moe_serve.gather(x, r, gw)
    place = got.place.cpu().long()
    flat = place[live].flatten()
    assert flat.unique().numel() == flat.numel() and bool((place[~live] == -1).all())
    assert bool((got.tile_group.cpu()[flat // 128] == ids[live].flatten()).all())
    assert torch.equal(got.rows[flat.to(DEV)], x[live.to(DEV)].repeat_interleave(s.top, 0))
    assert close(got.gate.double(), torch.sigmoid(x.double() @ gw.double()[0]), 1e-5)
    want = mixture_reference(x.double().cpu(), ids, r.weights.double().cpu(), gate_up.double().cpu(), down.double().cpu(), shared.double().cpu(),
                             gw[0].double().cpu()) if T <= 100 else None
    outs = []
    for kernel in ["general"] + (["tensor"] if dtype == torch.bfloat16 and d % 8 == 0 and F % 8 == 0 else []):
        y = moe_serve.product(moe_serve.glu(moe_serve.product(got.rows, gate_up, got, kernel), got), down, got, kernel)
        outs.append(moe_serve.combine(y, r, got, shared))
        if want is not None:
            assert close(outs[-1].double().cpu(), want, 2e-5 if dtype == torch.float32 else 2e-2), kernel
    assert all(close(o, outs[0], 2e-2) for o in outs)


@pytest.mark.parametrize("mixture", [dict(experts=8, top_k=2, expert_features=64, shared_features=48, shared_gate=True),
                                     dict(experts=16, top_k=4, expert_features=32, score_function="sigmoid", bias=True, groups=4, topk_groups=2, scaling=2.0)])
def test_served_layer_equals_the_training_layer(mixture):
    from dew_b200.models.causal_transformer import Mixture
    from dew_b200.nn.moe import SparseMLP
    torch.manual_seed(0)
    m = SparseMLP(128, Mixture(**mixture), 64, dtype=torch.bfloat16, device=DEV).eval()
    if m.router.expert_bias is not None:
        m.router.expert_bias.copy_(rnd(16) * 0.1)
    x = rnd(3, 50, 128, dtype=torch.bfloat16)
    with torch.no_grad():
        got, want = m(x, serving=True), m(x)
        # (a close call of the router may go the other way: the training layer's logits are the same sums in another order)
        bad = ((got - want).float().abs().amax(-1) > 2e-2 * want.float().abs().max()).float().mean()
        assert float(bad) < 0.02
        before = m.router.split()
        m.router.weight.mul_(2.0)
        assert not torch.equal(m.router.split().rows.float(), before.rows.float())


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_on_every_schedule(tmp_path, name, dtype):
    cfg, w, m = C.load(tmp_path, name, dtype, DEV)
    tokens = C.prompt(cfg, 150)
    want, _ = O.run(cfg, w, tokens)
    if dtype == torch.float32:
        bad = lambda got, ref=want: C.error(got, ref) > 2e-4
    else:
        # bf16 decides the router's close calls one way or the other, so a few positions may differ by an expert: nine in ten stay within what
        # rounding alone costs the plain PyTorch forms in bf16 on the CPU
        tol = 0.02 + 3 * float(C.row_errors(C.load(tmp_path / "cpu", name, dtype)[2](torch.tensor([tokens]))[0], want).quantile(0.6))
        bad = lambda got, ref=want: float((C.row_errors(got, ref) > tol).float().mean()) > 0.25 or tol > 0.4
    assert not bad(C.replay(m, [tokens]))
    for size in (2, 50, 64, 65):
        assert not bad(C.replay(m, C.cut(tokens, size), pool_tokens=160)), size
    assert not bad(C.replay(m, [tokens[:100]] + C.cut(tokens[100:], 1)))
    with torch.no_grad():
        assert not bad(m(torch.tensor([tokens], device=DEV))[0])
    if dtype == torch.bfloat16:
        return
    seqs = [C.prompt(cfg, n + 6, seed=n) for n in (1, 130, 40)]
    from dew_b200.sampling.text import RowBatch
    b = RowBatch(m, 3, 192, pool_tokens=300)
    for _ in range(2):
        b.feed([s[:-6] for s in seqs])
        for t in range(6, 0, -1):
            out = b.feed([[s[-t]] if t > 3 or i != 1 else [] for i, s in enumerate(seqs)], [[0] if t > 3 or i != 1 else [] for i in range(3)])
        alone = [C.replay(m, [s[:-6]] + C.cut(s[-6:], 1)) for s in seqs]
        assert C.error(out[0:1], alone[0][-1:].double().cpu()) < 2e-4 and C.error(out[1:2], alone[2][-1:].double().cpu()) < 2e-4
        for r in range(3):
            b.release(r)


def test_long_decoding_in_the_tensor_core_path(tmp_path):
    """bf16 decoding across chunk and page borders against the same positions of one prompt."""
    cfg, w, m = C.load(tmp_path, "wide", torch.bfloat16, DEV)
    tokens = C.prompt(cfg, 420)
    whole, steps = C.replay(m, [tokens]), C.replay(m, [tokens[:90]] + C.cut(tokens[90:], 1))
    e = C.row_errors(steps, whole.cpu())
    assert float(e.median()) < 0.05 and float((e > 0.3).float().mean()) < 0.1


def test_server_and_generate_agree(tmp_path):
    from dew_b200.inference import Server
    from dew_b200.sampling.text import Sampling, generate
    cfg, w, m = C.load(tmp_path, "wide", torch.float32, DEV)
    prompts = [C.prompt(cfg, n, seed=n) for n in (1, 70, 150, 33)]
    gen = generate(m, None, prompts, 8, sampling=Sampling(temperature=0.0))
    got = [gen.new_tokens(r).tolist() for r in range(4)]
    for p, g in zip(prompts, got):                                      # greedy under the restated decoder, token by token
        logits = O.run(cfg, w, p + g[:-1])[0][len(p) - 1:]
        top = logits.max(-1).values
        assert all(float(top[i] - logits[i, t]) < 1e-3 for i, t in enumerate(g))
    for graph in (False, True):
        server = Server(m, slots=2, capacity=192, kv_cache=KVCache(page_size=64), chunk=64, cuda_graph=graph)
        assert server(prompts, max_new_tokens=8) == got


@pytest.mark.parametrize("design", ["fakonex", "rotary"])
def test_decode_step_with_experts_replays_from_a_graph(tmp_path, design):
    """Rows whose positions change between replays, in bf16 with the paged decode kernels; the served experts also run under the decoders that were
    here before."""
    from dew_b200.inference import Server
    from dew_b200.models.causal_transformer import CausalTransformer, Mixture
    if design == "fakonex":
        cfg, w, m = C.load(tmp_path, "wide", torch.bfloat16, DEV)
    else:
        torch.manual_seed(0)
        cfg = {"vocab": 64}
        m = CausalTransformer(vocab_size=64, emb_features=256, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=128, max_seq_len=256, qk_norm=False,
                              mixture=Mixture(experts=8, top_k=2, expert_features=64), dtype=torch.bfloat16, device=DEV).eval()
        for p in m.parameters():
            p.requires_grad_(False)
    prompts = [C.prompt(cfg, n, seed=n) for n in (5, 90, 129)]
    runs = [Server(m, slots=4, capacity=256, kv_cache=KVCache(page_size=64), cuda_graph=g)(prompts, max_new_tokens=12) for g in (False, True)]
    assert runs[0] == runs[1]
