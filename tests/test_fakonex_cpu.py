"""The Fakonex design on the CPU: every mechanism against its plain restatement, whole models against the restated decoder, the cached paths
(token by token, portions, batches, re-used rows and pages), generation through both entry points, and the release format."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import fakonex_cases as C
import fakonex_oracle as O

from dew_b200.interop.hf import Pretrained
from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore
from dew_b200.ops import moe_serve, paged, streams
from dew_b200.sampling.text import RowBatch, Sampling, generate

D64 = torch.float64
TOL = 1e-4          # fp32 rounding through layers that normalise small vectors; a fault of any mechanism is past 1e-2


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("n", [1, 3])
def test_a_sub_layers_output_is_normalised_before_it_joins(n):
    T, d = 4, 10
    H, y, w, wy = rnd(T, n, d, seed=1), 7 * rnd(T, d, seed=2), rnd(d, seed=3), rnd(d, seed=4)
    got, H2 = streams.stream_step(H.clone(), streams.Write(y, weight=wy, eps=0.3), None, w, 0.2, torch.float32, "rms")
    for t in range(T):
        new = H[t].to(D64) + O.rms_norm(y[t].to(D64), wy.to(D64), 0.3)
        assert torch.allclose(H2[t].to(D64), new, atol=1e-5)
        assert torch.allclose(got[t].to(D64), O.rms_norm(new.sum(0), w.to(D64), 0.2), atol=1e-5)


@pytest.mark.parametrize("heads", [paged.Heads(4, 2, 8, 5, True, True), paged.Heads(3, 1, 6, 9, True, False), paged.Heads(5, 1, 7, 7, False, True)])
def test_heads_are_normalised_one_by_one_after_the_bias(heads):
    H, G, dk, dv = heads
    qkv, b, qw, kw = rnd(2, 3, heads.row), rnd(heads.packed, seed=1), rnd(dk, seed=2), rnd(dk, seed=3)
    q, k, v = paged.prepare_reference(qkv, heads, qw, kw if heads.own else None, 0.1, None, torch.arange(3)[None].expand(2, 3), b)
    for r in range(2):
        for t in range(3):
            x = (qkv[r, t, :heads.packed] + b).to(D64)
            assert torch.allclose(q[r, t].to(D64), O.head_norm(x[:H * dk], H, qw.to(D64), 0.1), atol=1e-5)
            if heads.own:
                assert torch.allclose(k[r, t].to(D64), O.head_norm(x[H * dk:(H + G) * dk], G, kw.to(D64), 0.1), atol=1e-5)
                assert torch.allclose(v[r, t].to(D64), x[(H + G) * dk:].view(G, dv), atol=1e-6)
    assert heads.own or (k is None and v is None)


@pytest.mark.parametrize("chunk", [1, 5, 8, 12, 40, None])
@pytest.mark.parametrize("heads", [paged.Heads(4, 2, 8, 5), paged.Heads(3, 1, 6, 9)])
def test_a_query_sees_its_own_chunk_and_nothing_before_it(heads, chunk):
    """Keys sit in shuffled pages; one key at a time is made to stand out for the last query: just inside and just outside its chunk, at page
    borders, at the first token."""
    T, page = 31, 8
    H, G, dk, dv = heads
    table = torch.tensor([[5, 0, 3, 7], [2, 6, 4, 8]], dtype=torch.int32)
    sinks = rnd(H, seed=5)
    lo = O.first_visible(T - 1, chunk)
    for target in sorted({0, 7, 8, T - 1, lo, max(lo - 1, 0), min(lo + 1, T - 1)}):
        qkv = rnd(2, T, heads.packed, seed=target)
        q, k = qkv[..., :H * dk], qkv[..., H * dk:(H + G) * dk]
        k[0, target] = 12 * torch.nn.functional.normalize(k[0, target], dim=-1)
        q[0, -1] = k[0, target].view(G, dk).repeat_interleave(H // G, 0).reshape(-1)
        pos = torch.arange(T, dtype=torch.int32)[None].repeat(2, 1)
        pages = paged.Pages(*(torch.full((10, page, G, max(dk, dv)), 99.0) for _ in range(2)), table, page, None)
        packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
        visible = paged.Visible(chunk, sinks)
        got = paged.paged_attend(packed[:, :, :H], heads, pos, pages, 0.5, visible=visible)
        one = paged.paged_attend(packed[:, -1:, :H], heads, pos[:, -1:].contiguous(), pages, 0.5, visible=visible)
        for r in range(2):
            split = [qkv[r, t].to(D64).split([H * dk, G * dk, G * dv]) for t in range(T)]
            qs, ks, vs = ([s[j].view(n, d) for s in split] for j, (n, d) in enumerate(((H, dk), (G, dk), (G, dv))))
            want = torch.stack(O.chunked_attention(qs, ks, vs, 0.5, chunk, sinks.to(D64)))
            assert torch.allclose(got[r].to(D64), want, atol=1e-4) and torch.allclose(one[r, 0].to(D64), want[-1], atol=1e-4)
        v = qkv[0, target, (H + G) * dk:].view(G, dv).repeat_interleave(H // G, 0)
        assert torch.allclose(got[0, -1], v, atol=0.2) == (target >= lo)                  # the planted key took the row, or is out of sight


def test_the_sink_counts_once_unscaled_and_per_head():
    s = torch.stack([rnd(1, 4, seed=h) for h in range(3)])[None]                          # [1, 3 heads, 1, 4]
    sinks = torch.tensor([-2.0, 0.0, 30.0])
    p = paged.softmax_with_sinks(s, sinks)
    for h in range(3):
        assert torch.allclose(p[0, h, 0].to(D64), O.sink_softmax(s[0, h, 0].to(D64), sinks[h].to(D64)), atol=1e-6)
    assert float(p[0, 2].sum()) < 1e-9 and float(paged.softmax_with_sinks(s, None).sum()) == pytest.approx(3.0)


def test_head_gates_read_the_last_columns_of_the_projection():
    o, z = rnd(2, 3, 4, 6), rnd(2, 3, 9, seed=1)
    got = paged.head_gate(o, z[..., 5:], 5)
    for h in range(4):
        assert torch.allclose(got[..., h, :].to(D64), o[..., h, :5].to(D64) * O.sigmoid(z[..., 5 + h].to(D64))[..., None], atol=1e-6)


@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (10, 3, 2, 1), (4, 2, 4, 2), (12, 3, 4, 1), (5, 5, 1, 1), (9, 1, 3, 3)])
def test_selection(E, top, groups, keep):
    z, b = rnd(40, E), rnd(E, seed=1) - 1.0
    s = moe_serve.Selection(E, top, groups, keep, float("-inf"), "sigmoid")
    w, ids, _ = moe_serve.select_reference(z, b, s)
    for t in range(40):
        chosen, weights = O.route(z[t].to(D64), b.to(D64), top, {"count": groups, "keep": keep} if groups > 1 else None)
        assert sorted(ids[t].tolist()) == sorted(chosen)
        assert torch.allclose(w[t][ids[t].argsort()].to(D64), weights[torch.tensor(chosen).argsort()], atol=1e-6)


def test_choice_scores_below_zero_do_not_let_a_dropped_group_back_in():
    z = torch.tensor([[0.0, 0.1, 5.0, -9.0]])
    b = torch.tensor([-2.0, -2.0, -1.5, -3.0])                        # the first group scores -2.97, the second -3.5; all choices are negative
    s = moe_serve.Selection(4, 2, 2, 1, float("-inf"), "sigmoid")
    assert sorted(moe_serve.select_reference(z, b, s)[1][0].tolist()) == [0, 1]
    assert sorted(O.route(z[0].to(D64), b.to(D64), 2, {"count": 2, "keep": 1})[0]) == [0, 1]
    # a fill of 0 (another design's rule) chooses the dropped ones here
    assert sorted(moe_serve.select_reference(z, b, s._replace(fill=0.0))[1][0].tolist()) == [2, 3]


def test_router_weights_split_into_bf16_rows():
    w = rnd(5, 16)
    exact = moe_serve.split_weights(w.to(torch.bfloat16).float())
    assert exact.exact and exact.rows.shape == (5, 16)
    two = moe_serve.split_weights(w)
    assert not two.exact and two.rows.shape == (13, 16) and bool((two.rows[5:8] == 0).all())
    assert torch.allclose(two.rows[:5].float() + two.rows[8:].float(), w, rtol=2e-5, atol=1e-7)


@pytest.mark.parametrize("name", ["plain", "odd"])
def test_expert_mixture(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    w = {k: v.to(D64) for k, v in w.items()}
    x = rnd(7, cfg["width"])
    for i, layer in enumerate(cfg["layers"]):
        if layer["mlp"]:
            want = torch.stack([O.expert_mixture(h.to(D64), w, f"l{i}.mlp.", layer["mlp"]) for h in x])
            assert torch.allclose(m.layers[i].mlp(x).to(D64), want, atol=1e-4 * float(want.abs().max()))


def test_softcap():
    x = 30 * rnd(3, 5)
    assert torch.allclose(streams.softcap(x, 6.0).to(D64), 6 * torch.tanh(x.to(D64) / 6), atol=1e-5)


def test_a_layer_that_shares_keys_reads_the_other_layers_pool():
    slots = [CacheSlot(2, 8, 8), CacheSlot(2, 8, 8, source=0), CacheSlot(1, 4, 4)]
    store = KVStore(KVCache(page_size=8, pages=4), 3, 1, 32, 0, 0, torch.float32, "cpu", slots=slots)
    assert store.k[1] is store.k[0] and store.v[1] is store.v[0] and store.k[2] is not store.k[0]
    with pytest.raises(ValueError):
        KVStore(KVCache(page_size=8), 2, 1, 32, 0, 0, torch.float32, "cpu", slots=[CacheSlot(2, 8, 8, source=1), CacheSlot(2, 8, 8)])
    with pytest.raises(ValueError):                                   # a projection with keys does not fit a slot without
        store.attend_slot(1, rnd(1, 2, 64), paged.Heads(4, 2, 8, 8), torch.arange(2)[None], scale=1.0)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_matches_the_restated_decoder(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    tokens = C.prompt(cfg, 70)
    want, layers = O.run(cfg, w, tokens)
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


@pytest.mark.parametrize("part", ["sink", "g", "q.norm", "k.norm", "q.b", "k.b", "v.b", "norm1b", "norm2b", "correction", "shared.sg", "router"])
def test_every_tensor_moves_the_logits(tmp_path, part):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    name = next(k for k in w if k.endswith("." + part))
    other = {**w, name: (w[name].float().roll(1, 0) * 1.5 + (0.5 if part == "shared.sg" else 0)).to(torch.bfloat16)}
    a = Pretrained.load(C.write(tmp_path / "a", cfg, w), dtype=torch.float32)
    b = Pretrained.load(C.write(tmp_path / "b", cfg, other), dtype=torch.float32)
    tokens = C.prompt(cfg, 30)
    with torch.no_grad():
        assert C.error(b(torch.tensor([tokens]))[0], a(torch.tensor([tokens]))[0]) > 1e-2
        assert C.error(b(torch.tensor([tokens]))[0], O.run(cfg, other, tokens)[0]) < TOL


def test_nothing_from_before_the_chunk_reaches_a_token(tmp_path):
    """Every layer in chunks of six: replacing the whole past outside the chunk changes nothing, replacing its first token does - in a prompt, in
    portions that cut the chunk, and decoded."""
    cfg, w, m = C.load(tmp_path, "sealed")
    tokens = C.prompt(cfg, 29)
    outside = [(t + 1) % cfg["vocab"] for t in tokens[:24]] + tokens[24:]
    inside = tokens[:24] + [(tokens[24] + 1) % cfg["vocab"]] + tokens[25:]
    for pieces in (lambda t: [t], lambda t: C.cut(t, 5), lambda t: [t[:22]] + C.cut(t[22:], 1), lambda t: C.cut(t, 2)):
        base = C.replay(m, pieces(tokens))
        assert torch.allclose(C.replay(m, pieces(outside))[24:], base[24:], atol=1e-5)
        assert bool(((C.replay(m, pieces(inside))[24:] - base[24:]).abs().amax(-1) > 1e-3).all())
        assert bool(((C.replay(m, pieces(outside))[18:24] - base[18:24]).abs().amax(-1) > 1e-3).all())


def test_batches_of_unequal_rows_and_reused_rows(tmp_path):
    cfg, w, m = C.load(tmp_path, "odd")
    lengths = (1, 67, 20, 5)
    seqs = [C.prompt(cfg, n + 8, seed=n) for n in lengths]
    wants = [O.run(cfg, w, s)[0] for s in seqs]
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
    """Portions that start at different positions share a call: a fresh row beside one far into its sequence."""
    cfg, w, m = C.load(tmp_path, "plain")
    a, c = C.prompt(cfg, 90, 3), C.prompt(cfg, 40, 4)
    wa, wc = O.run(cfg, w, a)[0], O.run(cfg, w, c)[0]
    b = RowBatch(m, 2, 128)
    b.feed([a[:64], []])
    out = b.feed([a[64:77], c[:31]], [list(range(13)), list(range(31))])
    assert C.error(out[:13], wa[64:77]) < TOL and C.error(out[13:], wc[:31]) < TOL
    out = b.feed([a[77:79], c[31:40]], [[0, 1], list(range(9))])
    assert C.error(out[:2], wa[77:79]) < TOL and C.error(out[2:], wc[31:40]) < TOL


def test_long_decoding_passes_many_chunks(tmp_path):
    cfg, w, m = C.load(tmp_path, "odd")                               # (its last layer sees the whole row)
    tokens = C.prompt(cfg, 200)
    want = O.run(cfg, w, tokens)[0]
    assert C.error(C.replay(m, [tokens[:3]] + C.cut(tokens[3:], 1)), want) < TOL
    other = [(tokens[0] + 1) % cfg["vocab"]] + tokens[1:]
    assert C.error(C.replay(m, [other[:3]] + C.cut(other[3:], 1))[-1:], want[-1:]) > 1e-3


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
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    gen = generate(m, None, prompts, 6, sampling=Sampling(temperature=0.0))
    assert [gen.new_tokens(r).tolist() for r in range(3)] == want
    server = Server(m, slots=2, capacity=64, kv_cache=KVCache(page_size=8), chunk=7)       # prompts in portions, slots and pages re-used
    assert server(prompts + prompts[::-1], max_new_tokens=6) == want + want[::-1]
    assert server.ledger.available() == server.ledger.pages
    shared = prompts[2][:17] + prompts[1]                             # starts with two pages another prompt has left in the pool
    hits = server.ledger.hits
    assert server([shared], max_new_tokens=6) == [_greedy(cfg, w, shared, 6)] and server.ledger.hits > hits


def test_the_stack_trains_in_its_differentiable_form(tmp_path):
    cfg, _, m = C.load(tmp_path, "plain")
    for p in m.parameters():
        p.requires_grad_(True)
    m.train()
    tokens = torch.tensor([C.prompt(cfg, 40), C.prompt(cfg, 40, 2), C.prompt(cfg, 40, 3)])
    loss = torch.nn.functional.cross_entropy(m(tokens[:, :-1]).flatten(0, 1), tokens[:, 1:].flatten())
    loss.backward()
    missing = [n for n, p in m.named_parameters() if p.grad is None or not bool(torch.isfinite(p.grad).all())]
    assert not missing
    aux = m.pop_aux()
    assert sorted(aux["effects"]) == [f"layers.{i}.mlp.router.expert_bias" for i in range(2)]
    assert m.param_count(active=True) < m.param_count()


# ------------------------------------------------------------------------------------------------ release format
@pytest.mark.parametrize("name", ["odd", "single"])
def test_release_round_trip(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name, torch.bfloat16)
    Pretrained.save(m, tmp_path / "again")
    again = json.loads((tmp_path / "again" / "config.json").read_text())
    strip = lambda c: {**c, "layers": [{**l, "mlp": l["mlp"] or None} for l in c["layers"]]}
    assert strip(again) == strip(cfg)
    from dew_b200.interop.release import Release
    stored = Release(tmp_path / "again")
    assert set(stored) == set(w) and all(torch.equal(stored[k].float(), w[k].float()) for k in w)
    tokens = torch.tensor([C.prompt(cfg, 12)])
    assert torch.equal(Pretrained.load(tmp_path / "again", dtype=torch.float32)(tokens), Pretrained.load(tmp_path / "model", dtype=torch.float32)(tokens))


def test_layer_without_a_feed_forward_may_bring_its_norms(tmp_path):
    cfg, w = C.CASES["odd"], C.tensors(C.CASES["odd"])
    more = {**w, "l1.norm2": w["l1.norm1"], "l1.norm2b": w["l1.norm1"]}
    tokens = torch.tensor([C.prompt(cfg, 12)])
    a, b = (Pretrained.load(C.write(tmp_path / n, cfg, t), dtype=torch.float32) for n, t in (("a", w), ("b", more)))
    assert torch.equal(a(tokens), b(tokens))


def test_releases_that_do_not_fit_are_refused(tmp_path):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    with pytest.raises(KeyError):                                     # a layer that shares keys has no projection of them
        Pretrained.load(C.write(tmp_path / "a", cfg, {**w, "l1.mix.k": w["l0.mix.k"]}))
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "b", cfg, {k: v for k, v in w.items() if k != "l1.mix.sink"}))
    with pytest.raises(ValueError):
        Pretrained.load(C.write(tmp_path / "c", cfg, {**w, "l0.mlp.e1.up": w["l0.mlp.e1.up"][:5]}))
    for change in (lambda l: l[0].update(type="convolution"), lambda l: l[1]["mixer"].update(kv_from=1), lambda l: l[1]["mixer"].update(kv_heads=4),
                   lambda l: l[0]["mlp"].update(kind="dense")):
        bad = json.loads(json.dumps(cfg))
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
    built = lookup("fakonex", "model")(**cfg)
    assert built.config == Pretrained.load(tmp_path / "model").config and built.family == "fakonex"


def test_trace_run_replays_a_batch(tmp_path):
    cfg, w, _ = C.load(tmp_path, "single")
    a, c = C.prompt(cfg, 30, 5), C.prompt(cfg, 12, 6)
    wa, wc = O.run(cfg, w, a)[0], O.run(cfg, w, c)[0]
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
