"""The Ragenex design on the CPU: every mechanism against its plain restatement, whole models against the restated decoder, the cached
paths (token by token, portions, batches, re-used rows and pages), generation through both entry points, and the release format."""
import json
import math
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import ragenex_cases as C
import ragenex_oracle as O

from dew_b200.interop.hf import Pretrained
from dew_b200.nn.kv_cache import KVCache
from dew_b200.ops import decayed, paged, streams
from dew_b200.sampling.text import RowBatch, Sampling, generate, make_cache

D64 = torch.float64
TOL = 1e-4          # fp32 rounding through layers that normalise small vectors; a fault of any mechanism is past 1e-2


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("n", [1, 2, 5])
def test_stream_step_is_write_read_norm(n):
    T, d = 3, 12
    H, y, scale, w = rnd(T, n, d, seed=1), rnd(T, d, seed=2), rnd(d, seed=3), rnd(d, seed=4)
    mix, out, read = rnd(n, n, seed=5), rnd(n, seed=6), rnd(n, seed=7)
    got, H2 = streams.stream_step(H.clone(), streams.Write(y, scale, mix, out), read, w, 1e-3, torch.float32)
    for t in range(T):
        new = O.stream_write([H[t, s].to(D64) for s in range(n)], mix.to(D64), out.to(D64), (scale * y[t]).to(D64))
        assert torch.allclose(H2[t].to(D64), torch.stack(new), atol=1e-5)
        assert torch.allclose(got[t].to(D64), O.layer_norm(O.stream_read(new, read.to(D64)), w.to(D64), 1e-3), atol=1e-4)
    plain, same = streams.stream_step(H.clone(), None, read, w, 1e-3, torch.float32)
    assert torch.equal(same, H)
    assert torch.allclose(plain[0].to(D64), O.layer_norm(O.stream_read([H[0, s].to(D64) for s in range(n)], read.to(D64)), w.to(D64), 1e-3), atol=1e-4)
    rms, _ = streams.stream_step(H.clone(), None, read, w, 1e-3, torch.float32, norm="rms")
    assert torch.allclose(rms[0].to(D64), O.rms_norm(O.stream_read([H[0, s].to(D64) for s in range(n)], read.to(D64)), w.to(D64), 1e-3), atol=1e-4)


def test_stream_norm_subtracts_a_large_mean_and_keeps_eps_inside_the_root():
    H = 1e3 + rnd(1, 1, 64)
    got, _ = streams.stream_step(H, None, torch.ones(1), torch.ones(64), 1e-5, torch.float32)
    assert torch.allclose(got[0].to(D64), O.layer_norm(H[0, 0].to(D64), torch.ones(64, dtype=D64), 1e-5), atol=1e-4)
    tiny = 1e-3 * rnd(1, 1, 64)
    got, _ = streams.stream_step(tiny, None, torch.ones(1), torch.ones(64), 1e-2, torch.float32)
    assert torch.allclose(got[0].to(D64), O.layer_norm(tiny[0, 0].to(D64), torch.ones(64, dtype=D64), 1e-2), rtol=1e-4)


def test_clamped_glu_and_gated_norm():
    gu = 3 * rnd(5, 14)
    got = streams.clamped_glu(gu, 1.25)
    assert torch.allclose(got.to(D64), O.clamped_glu(gu[:, :7].to(D64), gu[:, 7:].to(D64), 1.25), atol=1e-5)
    edge = torch.tensor([[5.0, -5.0, 5.0, -5.0]])                      # the gate has no lower bound, the linear half has both
    assert torch.allclose(streams.clamped_glu(edge, 2.0)[0], torch.tensor([2 / (1 + math.exp(-3.404)) * 3, -5 / (1 + math.exp(8.51)) * -1]))
    x, g, w = rnd(4, 9), rnd(4, 9, seed=1), rnd(9, seed=2)
    got = streams.sigmoid_gated_norm(x, g, w, 1e-3)
    want = torch.stack([O.rms_norm(a.to(D64), w.to(D64), 1e-3) / (1 + torch.exp(-b.to(D64))) for a, b in zip(x, g)])
    assert torch.allclose(got.to(D64), want, atol=1e-5)


def test_query_temperature_steps():
    got = paged.query_temperature(torch.arange(40), 0.7, 6)
    assert torch.allclose(got.to(D64), torch.tensor([O.query_temperature(p, 0.7, 6) for p in range(40)], dtype=D64), atol=1e-6)
    assert got[4] == 1 and got[5] > 1 and got[10] == got[5] and got[11] > got[5]          # the step is where p + 1 is a multiple


@pytest.mark.parametrize("H,dk,dv", [(1, 4, 4), (3, 6, 10), (2, 16, 5)])
def test_decayed_attention_in_portions(H, dk, dv):
    T = 23
    x = rnd(2, T, H * (2 * dk + dv))
    decay = torch.tensor([0.0, 0.5, 1.0][:H])
    state = torch.full((4, H, dk, dv), 7.0)                           # what an earlier sequence left behind
    ids, out = torch.tensor([3, 1]), []
    pos = torch.arange(T)[None].repeat(2, 1)
    for a, b in ((0, 2), (2, 3), (3, 17), (17, 23)):
        out.append(decayed.decayed_attention(x[:, a:b], decay, H, dk, dv, state, pos[:, a:b], ids))
    got = torch.cat(out, 1)
    for r in range(2):
        q, k, v = (O.silu(t.to(D64)) for t in x[r].split([H * dk, H * dk, H * dv], -1))
        want, last = O.decayed_recurrence(list(q.view(T, H, dk)), list(k.view(T, H, dk)), list(v.view(T, H, dv)), decay.to(D64))
        assert torch.allclose(got[r].to(D64), torch.stack(want), atol=1e-4)
        assert torch.allclose(state[ids[r]].to(D64), last, atol=1e-4)
    assert bool((state[0] == 7).all()) and bool((state[2] == 7).all())


def test_decayed_attention_padding_changes_nothing():
    H, dk, dv = 2, 4, 6
    x, decay = rnd(2, 9, H * (2 * dk + dv)), torch.tensor([0.6, 0.9])
    pos = torch.full((2, 9), -1)
    pos[0, :5] = torch.arange(5)
    state = torch.full((2, H, dk, dv), 3.0)
    got = decayed.decayed_attention(x, decay, H, dk, dv, state, pos)
    alone = torch.zeros(1, H, dk, dv)
    want = decayed.decayed_attention(x[:1, :5], decay, H, dk, dv, alone, pos[:1, :5])
    assert torch.allclose(got[0, :5], want[0]) and torch.allclose(state[0], alone[0]) and bool((got[0, 5:] == 0).all())
    assert bool((state[1] == 3).all()) and bool((got[1] == 0).all())


@pytest.mark.parametrize("heads", [paged.Heads(4, 2, 8, 5), paged.Heads(3, 1, 6, 9)])
def test_paged_attention_sees_every_earlier_key_across_pages(heads):
    """Keys sit in shuffled pages; one key at a time is made to stand out for one query, at page borders and far back."""
    T, page = 37, 8
    H, G, dk, dv = heads
    table = torch.tensor([[5, 0, 3, 7, 1], [2, 6, 4, 8, 9]], dtype=torch.int32)
    for target in (0, 1, 7, 8, 9, 15, 16, 35, 36):
        qkv = rnd(2, T, heads.packed, seed=target)
        q, k = qkv[..., :H * dk], qkv[..., H * dk:(H + G) * dk]
        k[0, target] = 12 * torch.nn.functional.normalize(k[0, target], dim=-1)
        q[0, -1] = k[0, target].view(G, dk).repeat_interleave(H // G, 0).reshape(-1)
        pos = torch.arange(T, dtype=torch.int32)[None].repeat(2, 1)
        pools = [torch.full((11, page, G, max(dk, dv)), 99.0) for _ in range(2)]
        pages = paged.Pages(*pools, table, page, None)
        packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
        got = paged.paged_attend(packed[:, :, :H], heads, pos, pages, 0.5)
        one = paged.paged_attend(packed[:, -1:, :H], heads, pos[:, -1:].contiguous(), pages, 0.5)
        for r in range(2):
            ks = [t.view(G, dk).to(D64) for t in qkv[r, :, H * dk:(H + G) * dk]]
            vs = [t.view(G, dv).to(D64) for t in qkv[r, :, (H + G) * dk:]]
            want = torch.stack(O.softmax_attention([t.view(H, dk).to(D64) for t in qkv[r, :, :H * dk]], ks, vs, 0.5))
            assert torch.allclose(got[r].to(D64), want, atol=1e-4) and torch.allclose(one[r, 0].to(D64), want[-1], atol=1e-4)
        v = qkv[0, target, (H + G) * dk:].view(G, dv).repeat_interleave(H // G, 0)
        assert torch.allclose(got[0, -1], v, atol=0.2)                # the planted key took the row
        assert bool((pools[0][10] == 99).all())                       # no page outside the table was written


def test_q_and_k_are_normalised_over_all_heads_at_once():
    heads = paged.Heads(4, 2, 8, 8)
    qkv, qw, kw = rnd(1, 3, heads.packed), rnd(32, seed=1), rnd(16, seed=2)
    q, k, _ = paged.prepare_reference(qkv, heads, qw, kw, 1e-3, (0.5, 2), torch.arange(3)[None])
    for t in range(3):
        want = O.rms_norm(qkv[0, t, :32].to(D64), qw.to(D64), 1e-3) * O.query_temperature(t, 0.5, 2)
        assert torch.allclose(q[0, t].reshape(-1).to(D64), want, atol=1e-5)
        assert torch.allclose(k[0, t].reshape(-1).to(D64), O.rms_norm(qkv[0, t, 32:48].to(D64), kw.to(D64), 1e-3), atol=1e-5)


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
    assert len(seen) == len(layers) == len(m.runs())
    for a, b in zip(seen, layers):
        assert torch.allclose(a.to(D64), b, atol=1e-4 * float(b.abs().max()))
    for size in (1, 2, 3, 16, 33, 70):
        assert C.error(C.replay(m, C.cut(tokens, size)), want) < TOL, size
    assert C.error(C.replay(m, [tokens[:50]] + C.cut(tokens[50:], 1)), want) < TOL


def test_batches_of_unequal_rows_and_reused_rows(tmp_path):
    cfg, w, m = C.load(tmp_path, "looped")
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
    cfg, w, m = C.load(tmp_path, "front")
    a, c = C.prompt(cfg, 90, 3), C.prompt(cfg, 40, 4)
    wa, wc = O.run(cfg, w, a)[0], O.run(cfg, w, c)[0]
    b = RowBatch(m, 2, 128)
    b.feed([a[:64], []])
    out = b.feed([a[64:77], c[:31]], [list(range(13)), list(range(31))])
    assert C.error(out[:13], wa[64:77]) < TOL and C.error(out[13:], wc[:31]) < 1e-5
    out = b.feed([a[77:79], c[31:40]], [[0, 1], list(range(9))])
    assert C.error(out[:2], wa[77:79]) < TOL and C.error(out[2:], wc[31:40]) < TOL


def test_long_decoding_keeps_the_first_token_in_reach(tmp_path):
    cfg, w, m = C.load(tmp_path, "plain")
    tokens = C.prompt(cfg, 200)
    want = O.run(cfg, w, tokens)[0]
    got = C.replay(m, [tokens[:3]] + C.cut(tokens[3:], 1))
    assert C.error(got, want) < TOL
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
    cfg, w, m = C.load(tmp_path, "looped")
    prompts = [C.prompt(cfg, n, seed=n) for n in (1, 9, 26)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    gen = generate(m, None, prompts, 6, sampling=Sampling(temperature=0.0))
    assert [gen.new_tokens(r).tolist() for r in range(3)] == want
    server = Server(m, slots=2, capacity=64, kv_cache=KVCache(page_size=8), chunk=7)       # prompts in portions, slots and pages re-used
    assert server(prompts + prompts[::-1], max_new_tokens=6) == want + want[::-1]
    assert server.ledger.available() == server.ledger.pages


def test_looped_decoder_with_rotary_attention_decodes_with_a_cache_per_pass():
    from dew_b200.models.causal_transformer import CausalTransformer, Loop
    torch.manual_seed(0)
    m = CausalTransformer(vocab_size=31, emb_features=32, num_layers=4, num_heads=4, num_kv_heads=2, mlp_features=48, max_seq_len=64,
                          loop=Loop(steps=3, first=1, end=3)).eval()
    tokens = torch.randint(0, 31, (2, 12))
    with torch.no_grad():
        full = m(tokens)
        cache = make_cache(m, 2, 32)
        assert cache.layers == 1 + 2 * 3 + 1
        out = [m(tokens[:, :7], positions=torch.arange(7)[None].expand(2, 7), cache=cache)]
        out += [m(tokens[:, t:t + 1], positions=torch.full((2, 1), t), cache=cache) for t in range(7, 12)]
    assert torch.allclose(torch.cat(out, 1), full, atol=1e-4)


def test_the_stack_trains_in_its_differentiable_form(tmp_path):
    cfg, _, m = C.load(tmp_path, "plain")
    for p in m.parameters():
        p.requires_grad_(True)
    tokens = torch.tensor([C.prompt(cfg, 20)])
    loss = torch.nn.functional.cross_entropy(m(tokens[:, :-1]).flatten(0, 1), tokens[0, 1:])
    loss.backward()
    missing = [n for n, p in m.named_parameters() if p.grad is None or not bool(torch.isfinite(p.grad).all())]
    assert not missing


# ------------------------------------------------------------------------------------------------ release format
def test_release_round_trip(tmp_path):
    cfg, w, m = C.load(tmp_path, "looped")
    Pretrained.save(m.to(torch.bfloat16), tmp_path / "again")
    again = json.loads((tmp_path / "again" / "config.json").read_text())
    assert again["loop"] == cfg["loop"] and again["streams"] == cfg["streams"]
    from dew_b200.interop.release import Release
    stored = Release(tmp_path / "again")
    assert set(stored) == set(w) and all(torch.equal(stored[k].float(), w[k].float()) for k in w)
    tokens = torch.tensor([C.prompt(cfg, 12)])
    assert torch.equal(Pretrained.load(tmp_path / "again", dtype=torch.float32)(tokens), Pretrained.load(tmp_path / "model", dtype=torch.float32)(tokens))


def test_release_with_missing_or_unknown_tensors_is_refused(tmp_path):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "a", cfg, {**w, "l0.mix.sink": torch.ones(4)}))
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "b", cfg, {k: v for k, v in w.items() if k != "l1.mix.g"}))
    with pytest.raises(ValueError):
        Pretrained.load(C.write(tmp_path / "c", cfg, {**w, "pos": w["pos"][:100]}))
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "convolution"
    with pytest.raises(ValueError):
        Pretrained.load(C.write(tmp_path / "d", bad, w))


def test_command_line_and_registry(tmp_path, capsys):
    from dew_b200.cli.main import main
    from dew_b200.utils.registry import lookup
    cfg, w, _ = C.load(tmp_path, "plain")
    p = C.prompt(cfg, 5)
    assert main(["generate", str(tmp_path / "model"), "--ids", ",".join(map(str, p)), "--max-new-tokens", "4", "--dtype", "float32", "--cpu"]) == 0
    assert json.loads(capsys.readouterr().out) == {"prompt": p, "tokens": _greedy(cfg, w, p, 4)}
    built = lookup("ragenex", "model")(**cfg)
    assert built.config == Pretrained.load(tmp_path / "model").config and built.family == "ragenex"


def test_too_many_tokens_are_refused(tmp_path):
    cfg, _, m = C.load(tmp_path, "plain")
    b = RowBatch(m, 1, 8)
    b.feed([[1] * 8])
    with pytest.raises(ValueError):
        b.feed([[1]])
    with pytest.raises(ValueError):
        RowBatch(m, 1, 8).feed([[cfg["vocab"]]])


def test_trace_run_replays_a_batch(tmp_path):
    cfg, w, _ = C.load(tmp_path, "front")
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
    assert os.access(root / "bin" / "trace_run", os.X_OK)
