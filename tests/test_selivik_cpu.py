"""The Selivik design on the CPU: every mechanism against its plain restatement, whole models against the restated decoder, the cached paths (token by
token, portions, batches, re-used rows and pages), generation through both entry points, and the release format."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import selivik_cases as C
import selivik_oracle as O

from dew_b200.interop.hf import Pretrained
from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore, pool_width
from dew_b200.ops import latent, moe_serve, paged, rotary, streams
from dew_b200.sampling.text import RowBatch, Sampling, generate

D64 = torch.float64
TOL = 1e-4          # fp32 rounding through a few layers; a fault of any mechanism is past 1e-2


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("rot", [rotary.Rotary(8, 500.0), rotary.Rotary(6, 1e4, False, 2.5), rotary.Rotary(4, 300.0, True), rotary.Rotary(10, 1e6, True, 3.0)])
def test_rotation(rot):
    x, pos = rnd(2, 3, 4, 10), torch.tensor([[0, 1, 977], [12345, 400000, 7]])
    got = rotary.turn(x, rotary.angles(pos, rot), rot)
    pairs = O.neighbours(rot.dims) if rot.interleaved else O.halves(rot.dims)
    for r in range(2):
        for t in range(3):
            for h in range(4):
                want = O.rotate_pairs(x[r, t, h].to(D64), int(pos[r, t]), pairs, rot.base, rot.dims, rot.factor)
                assert torch.allclose(got[r, t, h].to(D64), want, atol=1e-6)
    with pytest.raises(ValueError):
        rotary.Rotary(5)


@pytest.mark.parametrize("heads,dims", [(paged.Heads(4, 2, 8, 5), 8), (paged.Heads(3, 1, 10, 7), 6)])
def test_heads_turn_and_then_lose_their_length(heads, dims):
    H, G, dk, dv = heads
    rot = rotary.Rotary(dims, 100.0, False, 2.0)
    qkv, b, pos = rnd(2, 3, heads.row), rnd(heads.packed, seed=1), torch.tensor([[0, 1, 2], [7, 8, 90]])
    q, k, v = paged.prepare_reference(qkv, heads, None, None, 0.1, None, pos, b, paged.Turned(rot, rotary.angles(pos, rot)), True)
    spec = {"dims": dims, "base": 100.0, "scaling": {"factor": 2.0}}
    for r in range(2):
        for t in range(3):
            x = (qkv[r, t] + b).to(D64)
            assert torch.allclose(q[r, t].to(D64), O.turned_heads(x[:H * dk], H, int(pos[r, t]), spec, 0.1), atol=1e-5)
            assert torch.allclose(k[r, t].to(D64), O.turned_heads(x[H * dk:(H + G) * dk], G, int(pos[r, t]), spec, 0.1), atol=1e-5)
            assert torch.allclose(v[r, t].to(D64), x[(H + G) * dk:].view(G, dv), atol=1e-6)


WINDOWS = [(5, 0), (5, 2), (1, 1), (8, 8), (3, 20), (40, 4), (None, 0)]


@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("heads", [paged.Heads(4, 2, 8, 5), paged.Heads(3, 1, 6, 9)])
def test_a_query_sees_its_window_and_the_kept_first_keys(heads, window, keep):
    """Keys sit in shuffled pages; one key at a time is made to stand out for the last query: just inside and just outside its window, at page
    borders, the last kept one and the one after it."""
    T, page = 31, 8
    H, G, dk, dv = heads
    table = torch.tensor([[5, 0, 3, 7], [2, 6, 4, 8]], dtype=torch.int32)
    sinks, cap = rnd(H, seed=5), 30.0
    lo = 0 if window is None else max(T - window, 0)
    for target in sorted({0, 7, 8, T - 1, lo, max(lo - 1, 0), max(keep - 1, 0), min(keep, T - 1)}):
        qkv = rnd(2, T, heads.packed, seed=target)
        q, k = qkv[..., :H * dk], qkv[..., H * dk:(H + G) * dk]
        k[0, target] = 12 * torch.nn.functional.normalize(k[0, target], dim=-1)
        q[0, -1] = k[0, target].view(G, dk).repeat_interleave(H // G, 0).reshape(-1)
        pos = torch.arange(T, dtype=torch.int32)[None].repeat(2, 1)
        pages = paged.Pages(*(torch.full((10, page, G, max(dk, dv)), 99.0) for _ in range(2)), table, page, None)
        packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
        visible = paged.Visible(None, sinks, window, keep, cap)
        got = paged.paged_attend(packed[:, :, :H], heads, pos, pages, 0.5, visible=visible)
        one = paged.paged_attend(packed[:, -1:, :H], heads, pos[:, -1:].contiguous(), pages, 0.5, visible=visible)
        for r in range(2):
            split = [qkv[r, t].to(D64).split([H * dk, G * dk, G * dv]) for t in range(T)]
            qs, ks, vs = ([s[j].view(n, d) for s in split] for j, (n, d) in enumerate(((H, dk), (G, dk), (G, dv))))
            want = torch.stack(O.attend(qs, ks, vs, 0.5, cap, window, keep, sinks.to(D64)))
            assert torch.allclose(got[r].to(D64), want, atol=1e-4) and torch.allclose(one[r, 0].to(D64), want[-1], atol=1e-4)
        v = qkv[0, target, (H + G) * dk:].view(G, dv).repeat_interleave(H // G, 0)
        assert torch.allclose(got[0, -1], v, atol=0.2) == (target in O.visible(T - 1, window, keep))      # it took the row, or is out of sight


def test_the_cap_bends_scores_and_leaves_the_sink_alone():
    heads, T = paged.Heads(2, 1, 4, 3), 6
    qkv, pos = 4 * rnd(1, T, heads.packed), torch.arange(T, dtype=torch.int32)[None]
    pages = paged.Pages(*(torch.zeros(2, 8, 1, 4) for _ in range(2)), torch.zeros(1, 1, dtype=torch.int32), 8, None)
    packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
    sinks = torch.tensor([5.0, -3.0])                                     # the first is past the cap: capping it too would show
    split = [qkv[0, t].to(D64).split([8, 4, 3]) for t in range(T)]
    qs, ks, vs = ([s[j].view(n, d) for s in split] for j, (n, d) in enumerate(((2, 4), (1, 4), (1, 3))))
    for cap in (0.0, 2.0):
        got = paged.paged_attend(packed[:, :, :2], heads, pos, pages, 0.7, visible=paged.Visible(sinks=sinks, softcap=cap))
        assert torch.allclose(got[0].to(D64), torch.stack(O.attend(qs, ks, vs, 0.7, cap, sinks=sinks.to(D64))), atol=1e-5)


def test_two_sub_layers_join_the_residual_together():
    T, d = 4, 10
    H, y, y2, s, s2, w = rnd(T, 1, d, seed=1), rnd(T, d, seed=2), rnd(T, d, seed=3), rnd(d, seed=4), rnd(d, seed=5), rnd(d, seed=6)
    got, H2 = streams.stream_step(H.clone(), streams.Write(y, s, y2=y2, scale2=s2, gain=0.3), None, w, 0.2, torch.float32, "rms", 1.0)
    for t in range(T):
        new = (H[t, 0] + 0.3 * (s * y[t] + s2 * y2[t])).to(D64)
        assert torch.allclose(H2[t, 0].to(D64), new, atol=1e-6)
        assert torch.allclose(got[t].to(D64), O.centred_norm(new, w.to(D64), 0.2), atol=1e-5)


def test_feed_forward_activation():
    gu = 3 * rnd(5, 12)
    want = O.gelu_tanh(gu[:, :6].to(D64)) * gu[:, 6:]
    assert torch.allclose(streams.gelu_glu(gu).to(D64), want, atol=1e-5)


@pytest.mark.parametrize("E,top", [(5, 2), (4, 1), (3, 3), (40, 6)])
def test_weights_are_the_softmax_over_the_chosen(E, top):
    z = 4 * rnd(30, E)
    z[0] -= 300                                                           # far from 0, and far apart
    z[1, 0] += 200
    w, ids, _ = moe_serve.select_reference(z, None, moe_serve.Selection(E, top, score="top_softmax"))
    for t in range(30):
        chosen, weights = O.route(z[t].to(D64), top)
        assert sorted(ids[t].tolist()) == sorted(chosen)
        assert torch.allclose(w[t][ids[t].argsort()].to(D64), weights[torch.tensor(chosen).argsort()], atol=1e-6)
    with pytest.raises(ValueError):
        moe_serve.select_reference(z, None, moe_serve.Selection(E, top, score="softmin"))


@pytest.mark.parametrize("name", ["plain", "odd"])
def test_expert_mixture(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    w = {k: v.to(D64) for k, v in w.items()}
    x = rnd(7, cfg["width"])
    for i, layer in enumerate(cfg["layers"]):
        if layer["mlp"]:
            want = torch.stack([O.feed_forward(h.to(D64), w, f"l{i}.mlp.", layer["mlp"]) for h in x])
            assert torch.allclose(m.layers[i].mlp(x).to(D64), want, atol=1e-4 * float(want.abs().max()))


LATENTS = [latent.Latent(3, 6, 4, 5, 10, 7, rotary.Rotary(4, 300.0, True)), latent.Latent(2, 5, 6, 9, 3, 4, rotary.Rotary(6, 50.0, True)),
           latent.Latent(1, 8, 2, 1, 16, 5, rotary.Rotary(2, 50.0, True))]


@pytest.mark.parametrize("lat", LATENTS)
def test_latent_attention_through_the_pages(lat):
    """Against the restated mixer, with one far key that stands out; a token leaves ``rank + rot_dim`` numbers and a decode step reads nothing else."""
    T, d, eps = 21, 12, 1e-3
    H = lat.heads
    m = {"heads": H, "dim": lat.dim, "rot_dim": lat.rot_dim, "vdim": lat.vdim, "kv_rank": lat.rank, "q_rank": lat.q_rank, "scale": 0.4,
         "rot": {"base": lat.rotary.base, "dims": lat.rot_dim}}
    w = {"dq": rnd(lat.q_rank, d), "dq.norm": 1 + 0.3 * rnd(lat.q_rank, seed=1), "uq": rnd(H * lat.width, lat.q_rank, seed=2), "dkv": rnd(lat.row, d, seed=3),
         "dkv.norm": 1 + 0.3 * rnd(lat.rank, seed=4), "uk": rnd(H * lat.dim, lat.rank, seed=5), "uv": rnd(H * lat.vdim, lat.rank, seed=6),
         "g": rnd(H * lat.vdim, d, seed=7), "o": torch.eye(H * lat.vdim)}
    x = rnd(T, d, seed=8)
    x[3] = 6 * x[3]
    want = torch.stack(O.latent_mixer(list(x.to(D64)), {k: v.to(D64) for k, v in w.items()}, "", m, eps))
    up = torch.cat([w["uk"].view(H, lat.dim, -1), w["uv"].view(H, lat.vdim, -1)], 1).reshape(-1, lat.rank)
    z = x @ torch.cat([w["dq"], w["dkv"], w["g"]]).t()
    slot = CacheSlot(1, lat.row, lat.rank, latent=True)
    for cuts in ([T], [1] * T, [13] + [1] * (T - 13), [2] * 10 + [1]):
        store = KVStore(KVCache(page_size=4, pages=8), 1, 2, 24, 0, 0, torch.float32, "cpu", slots=[slot])
        assert store.v[0] is store.k[0] and store.k[0].shape[-1] == pool_width(slot, torch.float32)
        store.page_table.copy_(torch.tensor([[5, 0, 3, 7, 1, 6], [2, 2, 2, 2, 2, 2]]))
        out, at = [], 0
        for n in cuts:
            pos = torch.stack([torch.arange(at, at + n), torch.full((n,), -1)])
            zz = torch.stack([z[at:at + n], torch.full((n, z.shape[1]), 9.0)])
            out.append(store.attend_latent(0, zz, lambda c: c @ w["uq"].t(), up, lat, pos, scale=0.4, eps=eps, q_weight=w["dq.norm"], kv_weight=w["dkv.norm"],
                                           gated=True)[0])
            at += n
        assert torch.allclose(torch.cat(out).to(D64), want, atol=2e-5 * float(want.abs().max()) + 1e-5)
        assert not bool(store.k[0][2].any())                              # the padded row's page


def test_partial_sums_settle_on_one_set_of_buffers():
    """Layers of different shapes take turns: the second pass finds what the first one left (a captured step must not lose its scratch)."""
    store = KVStore(KVCache(page_size=8), 1, 1, 32, 0, 0, torch.float32, "cpu", slots=[CacheSlot(1, 8, 8)])
    shapes = [(16 * 4, 64), (8 * 2, 256), (16 * 3, 512), (1000, 8)]
    for n, width in shapes:
        store._partials(n, width, "cpu")
    left = [t.data_ptr() for t in store._scratch]
    for n, width in shapes:
        a, b, c = store._partials(n, width, "cpu")
        assert a.numel() >= n and b.numel() >= n and c.numel() >= n * width
    assert [t.data_ptr() for t in store._scratch] == left


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_matches_the_restated_decoder(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    tokens, want, layers = C.wanted(name, 70)
    got = m(torch.tensor([tokens]))[0]
    assert C.error(got, want) < TOL
    seen = []
    m._static(torch.tensor([tokens]), None, None, observe=lambda r, total: seen.append(total[0].clone()))
    assert len(seen) == len(layers)
    for a, b in zip(seen, layers):
        assert torch.allclose(a.to(D64), b, atol=1e-4 * float(b.abs().max()))
    for size in (1, 2, 3, 16, 33, 70):
        assert C.error(C.replay(m, C.cut(tokens, size)), want) < TOL, size
    assert C.error(C.replay(m, [tokens[:50]] + C.cut(tokens[50:], 1)), want) < TOL


@pytest.mark.parametrize("part", ["l0.mix.sink", "l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.norm1", "l0.ls1", "l0.ls2", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l1.mix.uk",
                                  "l1.mix.uv", "l1.mix.g", "l1.mlp.router", "l1.mlp.router.b", "l1.mlp.e1.down", "final.norm", "l0.mlp.gate"])
def test_every_tensor_moves_the_logits(tmp_path, part):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    other = {**w, part: (w[part].float().roll(1, 0) * 1.5).to(torch.bfloat16)}
    tokens = C.prompt(cfg, 30)
    b = Pretrained.load(C.write(tmp_path / "b", cfg, other), dtype=torch.float32)
    want = O.run(cfg, other, tokens)[0]
    with torch.no_grad():
        assert C.error(b(torch.tensor([tokens]))[0], want) < TOL
    assert C.error(O.run(cfg, w, tokens)[0], want) > 5e-3


CHANGES = {"window one longer": lambda c: c["layers"][0]["mixer"]["mask"].update(size=8), "one more kept": lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=3),
           "one kept less": lambda c: c["layers"][2]["mixer"]["mask"].update(keep_first=4), "cap": lambda c: c["layers"][0]["mixer"].update(softcap=2.7),
           "scale": lambda c: c["layers"][0]["mixer"].update(scale=0.42), "factor": lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=2.2),
           "base": lambda c: c["layers"][0]["mixer"]["rot"].update(base=400.0), "turned part": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6),
           "latent scale": lambda c: c["layers"][1]["mixer"].update(scale=0.37), "latent base": lambda c: c["layers"][1]["mixer"]["rot"].update(base=200.0),
           "embedding": lambda c: c["embedding"].update(scale=3.1), "residual factor": lambda c: c.update(residual_mult=0.62), "eps": lambda c: c["norm"].update(eps=0.02),
           "experts chosen": lambda c: c["layers"][1]["mlp"]["router"].update(top=3)}


@pytest.mark.parametrize("change", sorted(CHANGES))
def test_every_constant_is_read(tmp_path, change):
    cfg = copy.deepcopy(C.CASES["plain"])
    CHANGES[change](cfg)
    w, tokens = C.tensors(C.CASES["plain"]), C.prompt(cfg, 40)
    m = Pretrained.load(C.write(tmp_path / "m", cfg, w), dtype=torch.float32).eval()
    want = O.run(cfg, w, tokens)[0]
    with torch.no_grad():
        assert C.error(m(torch.tensor([tokens]))[0], want) < TOL
        assert C.error(C.replay(m, [tokens[:20]] + C.cut(tokens[20:], 1)), want) < TOL
    assert C.error(C.wanted("plain", 40)[1], want) > 1e-3


def test_nothing_between_the_kept_keys_and_the_window_reaches_a_token(tmp_path):
    cfg, w, m = C.load(tmp_path, "sealed")                                # a window of six, two kept
    tokens = C.prompt(cfg, 29)
    other = lambda t: (t + 1) % cfg["vocab"]
    between = tokens[:2] + [other(t) for t in tokens[2:18]] + tokens[18:]
    last_kept, edge = tokens[:1] + [other(tokens[1])] + tokens[2:], tokens[:18] + [other(tokens[18])] + tokens[19:]
    for pieces in (lambda t: [t], lambda t: C.cut(t, 5), lambda t: [t[:20]] + C.cut(t[20:], 1), lambda t: C.cut(t, 2)):
        base = C.replay(m, pieces(tokens))
        moved = lambda t: (C.replay(m, pieces(t)) - base).abs().amax(-1)
        assert float(moved(between)[23:].max()) < 1e-5 and bool((moved(between)[3:23] > 1e-3).all())
        assert bool((moved(last_kept)[1:] > 1e-3).all())
        assert bool((moved(edge)[18:24] > 1e-3).all()) and float(moved(edge)[24:].max()) < 1e-5


@pytest.mark.parametrize("name", ["odd", "plain"])
def test_batches_of_unequal_rows_and_reused_rows(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    lengths = (1, 67, 20, 5)
    seqs, wants = zip(*((C.wanted(name, n + 8, seed=n)[:2]) for n in lengths))
    b = RowBatch(m, 4, 128, pool_tokens=200)
    for turn in range(2):                                             # the second turn runs on freed rows and pages, in another order
        order = [0, 1, 2, 3] if turn == 0 else [2, 0, 3, 1]
        out = b.feed([seqs[i][:lengths[i]] for i in order], [list(range(lengths[i])) for i in order])
        for i, part in zip(order, out.split([lengths[i] for i in order])):
            assert C.error(part, wants[i][:lengths[i]]) < TOL
        left = {i: 8 if i != 1 else 3 for i in order}                 # one row ends early and rests
        for step in range(8):
            on = [step < left[i] for i in order]
            out = b.feed([[seqs[i][lengths[i] + step]] if o else [] for i, o in zip(order, on)], [[0] if o else [] for o in on])
            for row, i in zip(out, [i for i, o in zip(order, on) if o]):
                assert C.error(row[None], wants[i][lengths[i] + step][None]) < TOL, (turn, i, step)
        for r in range(4):
            b.release(r)
        assert b.ledger.available() == b.ledger.pages


def test_rows_at_different_places_in_one_batch(tmp_path):
    cfg, w, m = C.load(tmp_path, "plain")
    (a, wa, _), (c, wc, _) = C.wanted("plain", 90, 3), C.wanted("plain", 40, 4)
    b = RowBatch(m, 2, 128)
    b.feed([a[:64], []])
    out = b.feed([a[64:77], c[:31]], [list(range(13)), list(range(31))])
    assert C.error(out[:13], wa[64:77]) < TOL and C.error(out[13:], wc[:31]) < TOL
    out = b.feed([a[77:79], c[31:40]], [[0, 1], list(range(9))])
    assert C.error(out[:2], wa[77:79]) < TOL and C.error(out[2:], wc[31:40]) < TOL


def test_long_decoding(tmp_path):
    cfg, w, m = C.load(tmp_path, "odd")                               # (some layers see the whole row)
    tokens, want, _ = C.wanted("odd", 180)
    assert C.error(C.replay(m, [tokens[:3]] + C.cut(tokens[3:], 1)), want) < TOL


# ------------------------------------------------------------------------------------------------ generation
def _greedy(cfg, w, tokens, n):
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(O.run(cfg, w, seq)[0][-1].argmax()))
    return seq[len(tokens):]


def test_greedy_generation_through_generate_and_the_server(tmp_path):
    from dew_b200.inference import Server
    cfg, w, m = C.load(tmp_path, "odd")
    prompts = [C.prompt(cfg, n, seed=n) for n in (1, 9, 26)]
    want = [_greedy(cfg, w, p, 5) for p in prompts]
    gen = generate(m, None, prompts, 5, sampling=Sampling(temperature=0.0))
    assert [gen.new_tokens(r).tolist() for r in range(3)] == want
    server = Server(m, slots=2, capacity=64, kv_cache=KVCache(page_size=8), chunk=7)       # prompts in portions, slots and pages re-used
    assert server(prompts + prompts[::-1], max_new_tokens=5) == want + want[::-1]
    assert server.ledger.available() == server.ledger.pages
    shared = prompts[2][:17] + prompts[1]                             # starts with two pages another prompt has left in the pool
    hits = server.ledger.hits
    assert server([shared], max_new_tokens=5) == [_greedy(cfg, w, shared, 5)] and server.ledger.hits > hits


def test_the_stack_trains_in_its_differentiable_form(tmp_path):
    cfg, _, m = C.load(tmp_path, "plain")
    for p in m.parameters():
        p.requires_grad_(True)
    m.train()
    tokens = torch.tensor([C.prompt(cfg, 40), C.prompt(cfg, 40, 2), C.prompt(cfg, 40, 3)])
    loss = torch.nn.functional.cross_entropy(m(tokens[:, :-1]).flatten(0, 1), tokens[:, 1:].flatten())
    loss.backward()
    assert not [n for n, p in m.named_parameters() if p.grad is None or not bool(torch.isfinite(p.grad).all())]
    assert m.pop_aux()["balance_loss"] is not None and m.param_count(active=True) < m.param_count()


# ------------------------------------------------------------------------------------------------ release format
@pytest.mark.parametrize("name", ["odd", "plain", "single"])
def test_release_round_trip(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name, torch.bfloat16)
    Pretrained.save(m, tmp_path / "again")
    assert json.loads((tmp_path / "again" / "config.json").read_text()) == cfg
    from dew_b200.interop.release import Release
    stored = Release(tmp_path / "again")
    assert set(stored) == set(w) and all(torch.equal(stored[k].float(), w[k].float()) for k in w)
    tokens = torch.tensor([C.prompt(cfg, 12)])
    assert torch.equal(Pretrained.load(tmp_path / "again", dtype=torch.float32)(tokens), Pretrained.load(tmp_path / "model", dtype=torch.float32)(tokens))


def test_releases_that_do_not_fit_are_refused(tmp_path):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "a", cfg, {**w, "l1.mix.k": w["l0.mix.k"]}))
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "b", cfg, {k: v for k, v in w.items() if k != "l0.mix.sink"}))
    for name in ("l1.mlp.e1.up", "l1.mix.uk", "l1.mix.dkv"):
        with pytest.raises(ValueError):
            Pretrained.load(C.write(tmp_path / "c", cfg, {**w, name: w[name][:5]}))
    for change in (lambda l: l[0].update(type="convolution"), lambda l: l[0]["mlp"].update(kind="sparse"), lambda l: l[0]["mixer"]["rot"].update(dims=9),
                   lambda l: l[1]["mixer"]["rot"].update(dims=20), lambda l: l[0]["mixer"]["rot"].update(scaling={"type": "yarn", "factor": 2.0})):
        bad = copy.deepcopy(cfg)
        change(bad["layers"])
        with pytest.raises(ValueError):
            Pretrained.load(C.write(tmp_path / "d", bad, w))


def test_command_line_and_registry(tmp_path, capsys):
    from dew_b200.cli.main import main
    from dew_b200.utils.registry import lookup
    cfg, w, _ = C.load(tmp_path, "plain")
    p = C.prompt(cfg, 5)
    assert main(["generate", str(tmp_path / "model"), "--ids", ",".join(map(str, p)), "--max-new-tokens", "4", "--dtype", "float32", "--cpu"]) == 0
    assert json.loads(capsys.readouterr().out) == {"prompt": p, "tokens": _greedy(cfg, w, p, 4)}
    built = lookup("selivik", "model")(**cfg)
    assert built.config == Pretrained.load(tmp_path / "model").config and built.family == "selivik"


def test_trace_run_replays_a_batch(tmp_path):
    cfg, w, _ = C.load(tmp_path, "single")
    (a, wa, _), (c, wc, _) = C.wanted("single", 30, 5), C.wanted("single", 12, 6)
    (tmp_path / "out").mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": c[:11], "want": [10, 0]}, {"id": "y", "tokens": a[:28], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": a[28:29], "want": [0]}, {"id": "x", "tokens": c[11:], "want": [0]}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": a[29:], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[:5], "want": [4]}], "end": ["x"]}]
    root = Path(__file__).resolve().parents[1]
    res = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out",
                          str(tmp_path / "out"), "--max-tokens", "64", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr
    assert res.stdout.split("\n")[:4] == [f"done {i}" for i in range(4)]
    got = [torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for i in range(4)]
    for g, want in zip(got, (wc[[10, 0]], torch.stack([wa[28], wc[11]]), wa[29:30], wa[4:5])):
        assert C.error(g, want) < TOL
