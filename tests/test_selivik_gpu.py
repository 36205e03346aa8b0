"""The Selivik design on a GPU: its kernels against the plain PyTorch forms, whole models in fp32 and bf16 against the restated decoder on every
schedule, and generation through both entry points (the server with its CUDA graph)."""
import pytest
import torch

import selivik_cases as C
import selivik_oracle as O

from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore, pool_width
from dew_b200.ops import latent, library, moe_serve, paged, rotary, streams

pytestmark = pytest.mark.gpu
DEV = "cuda"


def rnd(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype).to(DEV)


def close(got, want, rel):
    return got.shape == want.shape and float((got.float() - want.float()).abs().max()) <= rel * float(want.float().abs().max().clamp_min(1e-6))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d", [(1, 64), (1, 4096), (1, 1100), (1, 7), (1, 9000), (3, 260)])
def test_residual_step_of_two_sub_layers(dtype, n, d):
    rel = 1e-5 if dtype == torch.float32 else 1e-2
    T = 9
    H, y, y2, s, s2, w = rnd(T, n, d, seed=2), rnd(T, d, seed=3, dtype=dtype), rnd(T, d, seed=4, dtype=dtype), rnd(d, seed=5, dtype=dtype), rnd(d, seed=6, dtype=dtype), \
        rnd(d, seed=7, dtype=dtype)
    for write in (streams.Write(y, s, y2=y2, scale2=s2, gain=0.3), streams.Write(y, y2=y2), streams.Write(y, s, gain=2.0), streams.Write(y, None, y2=y2, scale2=s2)):
        for norm, around in (("rms", 1.0), ("rms", 0.0), ("layer", 0.0)):
            ref, H_ref = streams.stream_step_reference(H, write, None, w, 1e-2, dtype, norm, around)
            got, H_got = streams.stream_step(H.clone(), write, None, w, 1e-2, dtype, norm, around)
            assert close(H_got, H_ref, 1e-5) and close(got, ref, rel)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_gain_activation_and_angles(dtype):
    table, ids = rnd(50, 36, dtype=dtype), torch.randint(0, 50, (2, 7), device=DEV)
    assert torch.equal(streams.embed_streams(ids, None, table, None, 1, 3.5)[:, :, 0], table[ids].float() * 3.5)
    gu = 4 * rnd(33, 2 * 37, dtype=dtype)
    for g in (gu, gu[:, :64].contiguous()):
        assert close(streams.gelu_glu(g), streams.gelu_glu_reference(g.float()), 1e-5 if dtype == torch.float32 else 1e-2)
    pos = torch.tensor([[0, 5, -1], [70000, 1 << 20, 3]], device=DEV)
    for rot in (rotary.Rotary(12, 1e4, False, 3.0), rotary.Rotary(6, 500.0, True)):
        assert torch.allclose(rotary.angles(pos, rot).cpu(), rotary.angles_reference(pos.cpu(), rot), atol=1e-7)


HEADS = [(paged.Heads(5, 1, 96, 88), 96), (paged.Heads(8, 2, 64, 64), 32), (paged.Heads(6, 2, 128, 80), 64), (paged.Heads(12, 1, 24, 40), 24),
         (paged.Heads(2, 2, 200, 130), 8), (paged.Heads(3, 1, 7, 5), 4), (paged.Heads(4, 4, 128, 128), 128), (paged.Heads(2, 1, 600, 520), 64)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dims", HEADS)
def test_projection_epilogue_with_rotation(dtype, heads, dims):
    rel = 1e-5 if dtype == torch.float32 else 1e-2
    H, G, dk, dv = heads
    D = max(8, (max(dk, dv) + 7) // 8 * 8)
    qkv, bias, qw, kw = rnd(2, 37, heads.row, dtype=dtype), rnd(heads.packed, seed=1, dtype=dtype), rnd(dk, seed=2, dtype=dtype), rnd(dk, seed=3, dtype=dtype)
    pos = torch.stack([torch.arange(37), torch.cat([torch.arange(5, 25), torch.full((17,), -1)])]).to(torch.int32)
    table = torch.tensor([[3, 1, 7], [2, 8, 4]], dtype=torch.int32)
    for rot in (rotary.Rotary(dims, 100.0, False, 2.0), rotary.Rotary(dims, 100.0, True)):
        for weights, unit in (((None, None), True), ((qw, kw), False), ((None, None), False)):
            pools = [torch.zeros(9, 16, G, D, dtype=dtype, device=DEV) for _ in range(2)]
            turned = paged.Turned(rot, rotary.angles(pos.to(DEV), rot))
            got = paged.qk_norm_append(qkv, heads, *weights, 1e-2, None, pos.to(DEV), paged.Pages(*pools, table.to(DEV), 16, None), bias, turned, unit)
            cpu = [p.cpu().float().zero_() for p in pools]
            want = paged.qk_norm_append(qkv.cpu().float(), heads, *(None if t is None else t.cpu().float() for t in weights), 1e-2, None, pos,
                                        paged.Pages(*cpu, table, 16, None), bias.cpu().float(), paged.Turned(rot, rotary.angles_reference(pos, rot)), unit)
            assert close(got.cpu(), want, rel)
            assert all(close(a.cpu(), b, rel) for a, b in zip(pools, cpu))


@pytest.mark.parametrize("S,D,Hq,Hkv,window,keep,cap", [(512, 128, 4, 2, 96, 3, 20.0), (512, 128, 4, 1, 128, 130, 0.0), (640, 64, 2, 2, 300, 1, 5.0), (384, 64, 3, 1, 1, 64, 0.0),
                                                       (1280, 128, 2, 1, 500, 0, 30.0), (1280, 128, 2, 1, 129, 300, 2.0)])
def test_flash_forward_with_kept_keys_and_cap(S, D, Hq, Hkv, window, keep, cap):
    from dew_b200.nn.kv_cache import visible_attention
    from dew_b200.ops.flash import Variants, flash_fwd
    q, k, v = (rnd(2, S, h, D, seed=i, dtype=torch.bfloat16) for i, h in enumerate((Hq, Hkv, Hkv)))
    q = q * 2
    sinks = rnd(Hq, seed=5) + 1
    for s in (None, sinks):
        got, lse = flash_fwd(q, k, v, True, 0.1, var=Variants(window, cap, s, keep=keep))
        want = visible_attention(q.float(), k.float(), v.float(), 0.1, paged.Visible(None, s, window, keep, cap))
        assert close(got, want, 1.5e-2) and bool(torch.isfinite(lse).all())


WINDOWS = [(1, 0), (1, 70), (48, 2), (64, 64), (100, 1), (129, 65), (257, 20), (None, 0)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("heads,dims", HEADS)
def test_attention_from_the_packed_projection(dtype, heads, dims, window, keep):
    """``attend_slot``: a prompt, portions at mixed positions, and decode steps, with planted keys just inside and just outside the window, the last
    kept key and the one after it, and at page borders."""
    rel = 2e-5 if dtype == torch.float32 else 6e-2      # bf16 queries and keys under sharp scores; a missed key is past 0.2
    H, G, dk, dv = heads
    rows, first, T = 3, 128, 300
    rot = rotary.Rotary(dims, 100.0, False, 3.0)
    kw = dict(scale=dk ** -0.5, eps=1e-3, bias=0.3 * rnd(heads.packed, seed=4, dtype=dtype), sinks=rnd(H, seed=5, dtype=dtype), window=window, keep=keep, softcap=9.0,
              rot=rot, unit=True)
    slots = [CacheSlot(G, dk, dv)]
    store = KVStore(KVCache(page_size=64, pages=24), 1, rows, 320, 0, 0, dtype, DEV, slots=slots)
    store.page_table.copy_(torch.randperm(24, generator=torch.Generator().manual_seed(0))[:15].reshape(3, 5).to(DEV))
    cpu = KVStore(KVCache(page_size=64, pages=24), 1, rows, 320, 0, 0, torch.float32, "cpu", slots=slots)
    cpu.page_table.copy_(store.page_table.cpu())
    ckw = {k: v.float().cpu() if isinstance(v, torch.Tensor) else v for k, v in kw.items()}
    x = rnd(rows, T, heads.row, seed=3, dtype=dtype)
    x[..., :(H + G) * dk] *= 3
    # a query that points at one key: rotated back by the distance between them
    back = lambda t, target, at: rotary.turn(rotary.turn(t[None], rotary.angles_reference(torch.tensor([target]), rot), rot) * 1.0,
                                             rotary.angles_reference(torch.tensor([at]), rot) * torch.tensor([1.0, -1.0]), rot)[0]
    k = (x[..., H * dk:(H + G) * dk] + kw["bias"][H * dk:(H + G) * dk]).cpu()
    for at in range(130, T, 13):
        lo = 0 if window is None else max(at - window + 1, 0)
        targets = ((lo, max(lo - 1, 0), min(at, at // 64 * 64)) if at % 2 else (max(keep - 1, 0), min(keep, at), lo))
        for r, target in enumerate(targets):
            q = back(k[r, target].view(G, dk).float(), target, at).repeat_interleave(H // G, 0)
            x[r, at, :H * dk] = (4 * q.reshape(-1)).to(dtype).to(DEV) - kw["bias"][:H * dk]

    def both(b, starts):
        n = max(e - s for s, e in zip(starts, b))
        xs, pos = torch.zeros(rows, n, heads.row, dtype=dtype, device=DEV), torch.full((rows, n), -1)
        for r in range(rows):
            xs[r, :b[r] - starts[r]] = x[r, starts[r]:b[r]]
            pos[r, :b[r] - starts[r]] = torch.arange(starts[r], b[r])
        got = store.attend_slot(0, xs, heads, pos.to(DEV), **kw)
        want = cpu.attend_slot(0, xs.float().cpu(), heads, pos, **ckw)
        for r in range(rows):
            m = b[r] - starts[r]
            assert m == 0 or close(got[r, :m].cpu(), want[r, :m], rel), (starts, b, r)
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


@pytest.mark.parametrize("D,Hq,Hkv", [(128, 8, 2), (128, 16, 1), (64, 8, 2), (256, 4, 2)])
def test_decode_in_windows_over_long_rows(D, Hq, Hkv):
    """Rows at and around window borders, with windows of many tiles (the balanced kernel cuts them into parts), kept keys of several tiles, and rows
    shorter than either."""
    heads = paged.Heads(Hq, Hkv, D, D)
    lens = [1, 64, 130, 1000, 1001, 2000, 2001, 2999, 4000, 4064]
    store = KVStore(KVCache(page_size=64), 1, len(lens), 4096, 0, 0, torch.bfloat16, DEV, slots=[CacheSlot(Hkv, D, D)])
    store.k[0].copy_(rnd(*store.k[0].shape, seed=1)), store.v[0].copy_(rnd(*store.v[0].shape, seed=2))
    for window, keep, cap in ((1000, 3, 20.0), (512, 200, 0.0), (96, 64, 4.0), (None, 0, 20.0), (1, 1, 0.0)):
        qkv, pos = rnd(len(lens), 1, heads.packed, seed=3, dtype=torch.bfloat16), torch.tensor(lens, device=DEV)[:, None] - 1
        sinks = rnd(Hq, seed=6)
        got = store.attend_slot(0, qkv, heads, pos, scale=0.2, window=window, keep=keep, softcap=cap, sinks=sinks)
        pages = paged.Pages(store.k[0].float(), store.v[0].float(), store.page_table, 64, None)
        want = paged.paged_attend_reference(qkv[..., :Hq * D].view(len(lens), 1, Hq, D).float(), heads, pos.int(), pages, 0.2,
                                            paged.Visible(None, sinks, window, keep, cap))
        assert close(got, want, 1.5e-2), (window, keep, cap)


# ------------------------------------------------------------------------------------------------ latent attention
def lat(heads, dim, rot, vdim, rank, q_rank, interleaved=True):
    return latent.Latent(heads, dim, rot, vdim, rank, q_rank, rotary.Rotary(rot, 200.0, interleaved))


LATENTS = [lat(3, 64, 32, 64, 96, 40), lat(5, 48, 16, 40, 56, 24), lat(2, 128, 64, 128, 512, 64), lat(20, 64, 16, 64, 256, 48), lat(2, 7, 6, 5, 11, 9),
           lat(33, 32, 8, 72, 40, 16), lat(1, 128, 32, 48, 128, 128, False), lat(4, 100, 20, 30, 50, 13), lat(2, 16, 8, 16, 640, 16), lat(2, 16, 8, 16, 1030, 16)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("l", LATENTS)
@pytest.mark.parametrize("page", [64, 16])
def test_latent_attention_on_every_schedule(dtype, l, page):
    """A prompt, later portions (rows that start together, and at different places), and decode steps, with queries that point at one far token."""
    rel = 3e-5 if dtype == torch.float32 else 6e-2
    rows, T = 3, 300
    slots = [CacheSlot(1, l.row, l.rank, latent=True)]
    n_pages = 24 * 64 // page
    store = KVStore(KVCache(page_size=page, pages=n_pages), 1, rows, 320, 0, 0, dtype, DEV, slots=slots)
    store.page_table.copy_(torch.randperm(n_pages, generator=torch.Generator().manual_seed(0))[:rows * (320 // page)].reshape(rows, -1).to(DEV))
    cpu = KVStore(KVCache(page_size=page, pages=n_pages), 1, rows, 320, 0, 0, torch.float32, "cpu", slots=slots)
    cpu.page_table.copy_(store.page_table.cpu())
    z = rnd(rows, T, l.q_rank + l.row + l.heads * l.vdim, seed=1, dtype=dtype)
    w, cw = 1 + 0.3 * rnd(l.q_rank, seed=2, dtype=dtype), 1 + 0.3 * rnd(l.rank, seed=3, dtype=dtype)
    uq, up = rnd(l.heads * l.width, l.q_rank, seed=4, dtype=dtype) * l.q_rank ** -0.5, rnd(l.heads * (l.dim + l.vdim), l.rank, seed=5, dtype=dtype) * l.rank ** -0.5
    kw = dict(scale=2.0 * l.width ** -0.5, eps=1e-3, gated=True)

    def both(b, starts, together=None):
        n = max(e - s for s, e in zip(starts, b))
        n = n if n == 1 else (n + 127) // 128 * 128
        zs, pos = torch.zeros(rows, n, z.shape[-1], dtype=dtype, device=DEV), torch.full((rows, n), -1)
        for r in range(rows):
            zs[r, :b[r] - starts[r]] = z[r, starts[r]:b[r]]
            pos[r, :b[r] - starts[r]] = torch.arange(starts[r], b[r])
        store.chunk_span = None if together is None else (starts[0] if together else 1, max(b))
        store.together = bool(together)
        got = store.attend_latent(0, zs, lambda c: torch.nn.functional.linear(c, uq), up, l, pos.to(DEV), q_weight=w, kv_weight=cw, **kw)
        want = cpu.attend_latent(0, zs.float().cpu(), lambda c: c @ uq.float().cpu().t(), up.float().cpu(), l, pos, q_weight=w.float().cpu(), kv_weight=cw.float().cpu(),
                                 **kw)
        for r in range(rows):
            m = b[r] - starts[r]
            assert m == 0 or close(got[r, :m].cpu(), want[r, :m], rel), (starts, b, r)
            assert bool(torch.isfinite(got[r]).all())

    at = [65, 64, 1]
    both(at, [0, 0, 0], True)
    both([66, 130, 1], at, False)                      # different places
    both([130, 130, 130], [66, 130, 1], False)
    both([258, 199, 130], [130, 130, 130], True)       # together, unequal ends
    at = [258, 199, 130]
    for t in range(42):
        nxt = [at[0] + 1, at[1] + (t % 3 > 0), at[2] + 1]
        both(nxt, at)
        at = nxt
    library.check_status()


@pytest.mark.parametrize("l", [x for x in LATENTS if x.rank <= 512])
def test_latent_kernels_agree(l):
    """The tensor-core and the general form against the latents, with one token that stands out for each row; several splits."""
    slot = CacheSlot(1, l.row, l.rank, latent=True)
    W = pool_width(slot, torch.bfloat16)
    R, S, T = 3, 2, 900
    store = KVStore(KVCache(page_size=64), 1, R, 960, 0, 0, torch.bfloat16, DEV, slots=[slot])
    store.k[0][..., :l.row] = rnd(*store.k[0].shape[:-1], l.row, seed=1)
    pages = paged.Pages(store.k[0], store.v[0], store.page_table, 64, None)
    pos = torch.tensor([[T - 2, T - 1], [63, 64], [-1, 0]], dtype=torch.int32, device=DEV)
    q = rnd(R, S, l.heads, W, seed=2, dtype=torch.bfloat16)
    q[..., l.row:] = 0
    flat = store.k[0].view(-1, W)
    for h in range(l.heads):                           # far tokens, page and tile borders
        at = (0, 31, 32, 63, 64, 500, T - 2)[h % 7]
        q[0, :, h] = 3 * flat[store.page_table[0, at // 64] * 64 + at % 64]
    got = latent.attend(q, l, pos, pages, 0.3, store.max_len)
    want = paged.paged_attend_reference(q.float(), paged.Heads(l.heads, 1, l.row, l.rank), pos, pages._replace(k=pages.k.float(), v=pages.v.float()), 0.3)
    assert close(got, want, 1.5e-2) and bool((got[2, 0] == 0).all())
    assert close(latent.attend(q, l, pos, pages, 0.3, store.max_len, kernel="general"), want, 1.5e-2)
    library.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("l", LATENTS)
@pytest.mark.parametrize("T", [1, 70])
def test_products_per_head(dtype, l, T):
    rel = 1e-5 if dtype == torch.float32 else 1e-2
    q, up = rnd(1, T, l.heads, l.width, dtype=dtype), rnd(l.heads * (l.dim + l.vdim), l.rank, seed=1, dtype=dtype)
    table = rotary.angles(torch.arange(T, device=DEV)[None] * 17, l.rotary)
    W = pool_width(CacheSlot(1, l.row, l.rank, latent=True), dtype)
    assert close(latent.absorb(q, up, l, table, W).cpu(), latent.absorb(q.cpu().float(), up.cpu().float(), l, table.cpu(), W), rel)
    o, z = rnd(1, T, l.heads, l.rank, seed=2, dtype=dtype), rnd(1, T, 3 + l.heads * l.vdim, seed=3, dtype=dtype)
    for gate in (None, z[..., 3:]):
        assert close(latent.expand(o, up, l, gate).cpu(), latent.expand(o.cpu().float(), up.cpu().float(), l, None if gate is None else gate.cpu().float()), rel)
    want = latent.rotate(q.cpu().float(), l, table.cpu())
    assert close(latent.rotate(q.clone(), l, table).cpu(), want, rel)


# ------------------------------------------------------------------------------------------------ the router
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d,E,top", [(1, 64, 8, 2), (37, 72, 5, 1), (70, 30, 6, 6), (600, 64, 200, 8), (700, 128, 300, 20)])
def test_softmax_over_the_chosen(dtype, T, d, E, top):
    s = moe_serve.Selection(E, top, score="top_softmax")
    x, b = rnd(T, d, dtype=dtype), 3 * rnd(E, seed=1)
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    pos[T // 2:T // 2 + T // 8] = -1
    live = (pos >= 0).cpu()
    for exact in (True, False):
        weight = 2 * d ** -0.5 * rnd(E, d, seed=2)
        weight = weight.to(torch.bfloat16).float() if exact else weight
        split = moe_serve.split_weights(weight)
        logits = (x.double() @ weight.double().t() + b.double()).cpu()
        for form in ["rows"] + (["product"] if dtype == torch.bfloat16 and d % 8 == 0 else []):
            r = moe_serve.route(x, weight, split if dtype == torch.bfloat16 else None, None, s, pos, kernel=form, logit_bias=b)
            ids = r.ids.cpu().long()
            assert bool((ids[~live] == -1).all()) and int(r.counts.sum()) == int(live.sum()) * top
            got = logits.gather(1, ids.clamp_min(0))
            assert bool((got[live] >= logits.topk(top, -1).values[:, -1:][live] - 2e-4).all()) and all(len(set(row)) == top for row in ids[live].tolist())
            assert close(r.weights.cpu()[live].double(), torch.softmax(got, -1)[live], 2e-5 if form == "rows" else 1e-4)
    with pytest.raises(ValueError):
        moe_serve.route(x, weight, None, None, s, pos[None, :0].reshape(-1), logit_bias=b)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_on_every_schedule(tmp_path, name):
    """fp32, every position."""
    cfg, w, m = C.load(tmp_path, name, torch.float32, DEV)
    tokens, want, _ = C.wanted(name, 150)
    good = lambda got, ref=want: C.error(got, ref) < 2e-4
    assert good(C.replay(m, [tokens]))
    for size in (2, 50, 64, 65):
        assert good(C.replay(m, C.cut(tokens, size), pool_tokens=160)), size
    assert good(C.replay(m, [tokens[:100]] + C.cut(tokens[100:], 1)))
    with torch.no_grad():
        assert good(m(torch.tensor([tokens], device=DEV))[0])


def tolerance(tmp_path, name, want, tokens):
    """What rounding alone costs the plain PyTorch forms in bf16 on the CPU, times three; every expert is chosen, so no close call adds to it."""
    cfg, _, m = C.load(tmp_path / "cpu", C.all_chosen(C.CASES[name]), torch.bfloat16)
    return 3 * C.error(m(torch.tensor([tokens]))[0], want)


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_bf16_model_on_every_schedule(tmp_path, name):
    """Every position of prompts, portions and decode steps, and a batch of unequal rows on re-used rows and pages."""
    tokens, want, _ = C.wanted(name, 150, sure=True)
    tol = tolerance(tmp_path, name, want, tokens)
    assert tol < 0.3
    cfg, w, m = C.load(tmp_path, C.all_chosen(C.CASES[name]), torch.bfloat16, DEV)
    good = lambda got, ref=want: C.error(got, ref) < tol
    assert good(C.replay(m, [tokens]))
    for size in (2, 50, 64, 65):
        assert good(C.replay(m, C.cut(tokens, size), pool_tokens=160)), size
    assert good(C.replay(m, [tokens[:60]] + C.cut(tokens[60:], 1)))
    from dew_b200.sampling.text import RowBatch
    lengths = (1, 130, 40)
    seqs, wants = zip(*(C.wanted(name, n + 6, seed=n, sure=True)[:2] for n in lengths))
    b = RowBatch(m, 3, 192, pool_tokens=300)
    for turn in range(2):
        order = [0, 1, 2] if turn == 0 else [2, 0, 1]
        out = b.feed([seqs[i][:lengths[i]] for i in order], [list(range(lengths[i])) for i in order])
        for i, part in zip(order, out.split([lengths[i] for i in order])):
            assert good(part, wants[i][:lengths[i]])
        for step in range(6):
            on = [step < 3 or i != 1 for i in order]
            out = b.feed([[seqs[i][lengths[i] + step]] if o else [] for i, o in zip(order, on)], [[0] if o else [] for o in on])
            for row, i in zip(out, [i for i, o in zip(order, on) if o]):
                assert good(row[None], wants[i][lengths[i] + step][None]), (turn, i, step)
        for r in range(3):
            b.release(r)
    library.check_status()


def test_long_decoding_in_the_tensor_core_path(tmp_path):
    """bf16 decoding across window and page borders against the same positions of one prompt."""
    cfg, w, m = C.load(tmp_path, C.all_chosen(C.CASES["wide"]), torch.bfloat16, DEV)
    tokens = C.prompt(cfg, 420)
    whole, steps = C.replay(m, [tokens]), C.replay(m, [tokens[:90]] + C.cut(tokens[90:], 1))
    portions = C.replay(m, C.cut(tokens, 128))
    assert C.error(steps, whole.cpu()) < 0.15 and C.error(portions, whole.cpu()) < 0.15


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
        for page in (64, 16):
            server = Server(m, slots=2, capacity=192, kv_cache=KVCache(page_size=page), chunk=64, cuda_graph=graph)
            assert server(prompts, max_new_tokens=8) == got


@pytest.mark.parametrize("page", [64, 16])
def test_decode_step_replays_from_a_graph(tmp_path, page):
    """Rows whose positions change between replays, in bf16 with the paged decode kernels; layers of both kinds share the scratch."""
    from dew_b200.inference import Server
    cfg, w, m = C.load(tmp_path, "wide", torch.bfloat16, DEV)
    prompts = [C.prompt(cfg, n, seed=n) for n in (5, 90, 129)]
    runs = [Server(m, slots=4, capacity=256, kv_cache=KVCache(page_size=page), cuda_graph=g)(prompts, max_new_tokens=12) for g in (False, True)]
    assert runs[0] == runs[1]
