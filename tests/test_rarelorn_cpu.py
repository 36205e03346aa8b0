"""The Rarelorn design on the CPU: every mechanism against its plain restatement, whole models against the restated decoder, the cached paths (token by
token, portions, batches, re-used rows and pages), generation through both entry points, and the release format."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import rarelorn_cases as C
import rarelorn_oracle as O

from dew_b200.interop.hf import Pretrained
from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore
from dew_b200.ops import moe_serve, paged, recurrence, streams, token_mix
from dew_b200.sampling.text import RowBatch, Sampling, generate

D64 = torch.float64
TOL = 1e-4          # fp32 rounding through a few layers; a fault of any mechanism is past 1e-2


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def rows_at(starts, ends, ids=None):
    """The rows of a call: row r brings its tokens ``[starts[r], ends[r])``."""
    n = max(1, max(e - s for s, e in zip(starts, ends)))
    pos = torch.full((len(starts), n), -1, dtype=torch.int32)
    for r, (s, e) in enumerate(zip(starts, ends)):
        pos[r, :e - s] = torch.arange(s, e)
    return token_mix.Rows(pos, (pos.amax(1) + 1).to(torch.int32), None if ids is None else torch.tensor(ids, dtype=torch.int32))


def pieces(x, starts, ends):
    """``x [R, T, C]`` cut to the tokens of a call, what lies past a row's end filled with noise."""
    n = max(1, max(e - s for s, e in zip(starts, ends)))
    out = 9 * torch.ones(x.shape[0], n, *x.shape[2:])
    for r, (s, e) in enumerate(zip(starts, ends)):
        out[r, :e - s] = x[r, s:e]
    return out


# portions of three rows (one rests at times), down to two tokens and one
SCHEDULE = [(9, 1, 0), (11, 3, 5), (12, 4, 6), (13, 4, 7), (17, 16, 9), (18, 17, 17)]


def on_schedule(call, want):
    """``call(rows, starts, ends)`` -> ``[3, n, ...]`` on every portion against ``want [3][T, ...]``; the rows lie shuffled in the store."""
    at = (0, 0, 0)
    for nxt in SCHEDULE:
        got = call(rows_at(at, nxt, [2, 0, 3]), at, nxt)
        for r in range(3):
            n = nxt[r] - at[r]
            assert torch.allclose(got[r, :n].to(D64), want[r][at[r]:nxt[r]], atol=2e-5, rtol=1e-5), (at, nxt, r)
            assert not got[r, n:].any()
        at = nxt


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("silu", [False, True])
def test_short_convolution(taps, silu):
    C_, T = 5, 18
    x, w, b = rnd(3, T, C_), rnd(C_, taps, seed=1), rnd(C_, seed=2)
    want = []
    for r in range(3):
        y = O.causal_conv([u.to(D64) for u in x[r] + b], w.to(D64))
        want.append(torch.stack([O.silu(v) if silu else v for v in y]))
    whole = token_mix.conv_tokens(x, w, b, silu)
    assert all(torch.allclose(whole[r].to(D64), want[r], atol=1e-5) for r in range(3))
    for _ in range(2):                                # (the second turn starts over what the first one left)
        state = 9 * torch.ones(4, C_, taps - 1)
        on_schedule(lambda rows, s, e: token_mix.conv_tokens(pieces(x, s, e), w, b, silu, rows, state), want)
    assert taps == 1 or bool((state[1] == 9).all())


def test_token_shift():
    d, T = 6, 18
    x, mu = rnd(3, T, d), torch.rand(4, d)
    want = [torch.stack([torch.stack(O.shifted([h.to(D64) for h in x[r]], m.to(D64))) for m in mu], 1) for r in range(3)]
    got = token_mix.shift_tokens(x, mu)
    assert all(torch.allclose(got[:, r].transpose(0, 1).to(D64), want[r], atol=1e-6) for r in range(3))
    state = 9 * torch.ones(4, d)
    on_schedule(lambda rows, s, e: token_mix.shift_tokens(pieces(x, s, e), mu, rows, state).permute(1, 2, 0, 3), want)


def test_low_rank_decay_and_gated_norms():
    z, w2, w0 = 2 * rnd(7, 5), rnd(9, 5, seed=1), rnd(9, seed=2)
    got = token_mix.low_rank_decay(z, w2, w0)
    for t in range(7):
        want = O.channel_decay(z[t].to(D64), torch.eye(5, dtype=D64), w2.to(D64), w0.to(D64))
        assert torch.allclose(got[t].to(D64).exp(), want, atol=1e-6)
    x, gate = rnd(2, 3, 4, 5), rnd(2, 3, 20, seed=1)
    for act, fn in (("silu", O.silu), ("sigmoid", O.sigmoid)):
        for w in (rnd(5, seed=3), rnd(20, seed=4)):
            got = token_mix.head_gated_norm(x, gate, w, 0.1, act)
            wide = w if w.numel() == 20 else w.repeat(4)
            for r in range(2):
                for t in range(3):
                    want = torch.cat([O.unit(h, 0.1) for h in x[r, t].to(D64)]) * wide.to(D64) * fn(gate[r, t].to(D64))
                    assert torch.allclose(got[r, t].to(D64), want, atol=1e-5)
    with pytest.raises(ValueError):
        token_mix.head_gated_norm(x, gate, w, 0.1, "relu")


def _delta_inputs(H, G, dk, dv, T=18):
    q, k, v, gates = rnd(3, T, G * dk), rnd(3, T, G * dk, seed=1), rnd(3, T, H * dv, seed=2), 2 * rnd(3, T, 2 * H, seed=3)
    return q, k, v, gates, rnd(H, seed=4) - 1, rnd(H, seed=5)


def _delta_wanted(q, k, v, gates, A_log, dt_bias, H, G, dk, dv):
    out = []
    for r in range(q.shape[0]):
        spread = lambda x: torch.stack([O.on_the_sphere(x.view(G, dk)[h // (H // G)].to(D64)) for h in range(H)])
        betas = [O.sigmoid(z[:H].to(D64)) for z in gates[r]]
        decays = [torch.exp(-torch.exp(A_log.to(D64)) * O.softplus(z[H:].to(D64) + dt_bias.to(D64))) for z in gates[r]]
        out.append(torch.stack(O.gated_delta([spread(x) * dk ** -0.5 for x in q[r]], [spread(x) for x in k[r]], [x.view(H, dv).to(D64) for x in v[r]], betas, decays)))
    return out


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 6, 9), (3, 3, 5, 4), (3, 1, 8, 8)])
def test_gated_delta_rule(H, G, dk, dv):
    q, k, v, gates, A_log, dt = _delta_inputs(H, G, dk, dv)
    q[0, 3], k[0, 3] = 0, 0                                             # a zero vector stays one
    want = _delta_wanted(q, k, v, gates, A_log, dt, H, G, dk, dv)
    got = recurrence.delta_rule(q, k, v, gates, A_log, dt, H, G)
    assert all(torch.allclose(got[r].to(D64), want[r], atol=1e-5) for r in range(3))
    for _ in range(2):
        state = 9 * torch.ones(4, H, dk, dv)
        on_schedule(lambda rows, s, e: recurrence.delta_rule(*(pieces(x, s, e) for x in (q, k, v, gates)), A_log, dt, H, G, None, rows, state), want)
    assert bool((state[1] == 9).all())


def test_a_delta_write_is_read_back_and_replaced():
    """Without decay and with whole steps the state is a table: the last value written under a key comes back, however far it lies."""
    H, dk, dv, T = 1, 8, 5, 40
    k = 0.01 * rnd(1, T, dk)
    k[..., 0] = 0
    k[:, 3], k[:, 9] = torch.eye(dk)[0] * 5, torch.eye(dk)[0] * 7        # the same direction twice
    q, v = k.clone(), rnd(1, T, dv, seed=1)
    q[:, -1] = torch.eye(dk)[0]
    gates = torch.cat([torch.full((1, T, 1), 30.0), torch.full((1, T, 1), -30.0)], -1)
    got = recurrence.delta_rule(q, k, v, gates, torch.zeros(1), torch.zeros(1), H, H, 1.0)
    assert torch.allclose(got[0, 3, 0], v[0, 3], atol=1e-3) and torch.allclose(got[0, 9, 0], v[0, 9], atol=1e-3)
    assert torch.allclose(got[0, -1, 0], v[0, 9], atol=1e-2)


def _memory_inputs(H, dk, dv, T=18):
    return rnd(3, T, H * dk), rnd(3, T, H * dk, seed=1), rnd(3, T, H * dv, seed=2), 3 * rnd(3, T, 2 * H, seed=3), rnd(H, seed=4), rnd(H, seed=5) + 1


def _memory_wanted(q, k, v, gates, bi, bf, H, dk, dv, cap):
    out = []
    for r in range(q.shape[0]):
        ins = [O.capped(z[:H].to(D64) + bi.to(D64), cap) for z in gates[r]]
        forgets = [O.log_sigmoid(O.capped(z[H:].to(D64) + bf.to(D64), cap)) for z in gates[r]]
        out.append(torch.stack(O.matrix_memory([x.view(H, dk).to(D64) * dk ** -0.5 for x in q[r]], [x.view(H, dk).to(D64) for x in k[r]],
                                               [x.view(H, dv).to(D64) for x in v[r]], ins, forgets)))
    return out


@pytest.mark.parametrize("H,dk,dv,cap", [(2, 6, 9, 4.0), (3, 5, 4, 15.0), (1, 8, 8, 0.7)])
def test_matrix_memory(H, dk, dv, cap):
    args = _memory_inputs(H, dk, dv)
    want = _memory_wanted(*args, H, dk, dv, cap)
    got = recurrence.matrix_memory(*args, H, cap)
    assert all(torch.allclose(got[r].to(D64), want[r], atol=2e-5, rtol=1e-4) for r in range(3))
    for _ in range(2):
        memory = recurrence.Memory(9 * torch.ones(4, H, dk, dv), 9 * torch.ones(4, H, dk), 9 * torch.ones(4, H))
        on_schedule(lambda rows, s, e: recurrence.matrix_memory(*(pieces(x, s, e) for x in args[:4]), *args[4:], H, cap, None, rows, memory), want)
    assert bool((memory.m[1] == 9).all())


def test_the_running_maximum_starts_at_zero_and_bounds_the_normaliser():
    """Input gates far below 0: the maximum stays at 0 and the denominator is exp(-m), so the outputs are as small as the gates say."""
    H, dk, dv, T, cap = 1, 4, 3, 5, 12.0
    q, k, v, gates, bi, bf = _memory_inputs(H, dk, dv, T)
    gates[..., 0] = -20.0
    got = recurrence.matrix_memory(q, k, v, gates, bi, bf, H, cap)
    want = _memory_wanted(q, k, v, gates, bi, bf, H, dk, dv, cap)
    assert all(torch.allclose(got[r].to(D64), want[r], rtol=1e-3, atol=1e-9) for r in range(3)) and float(got.abs().max()) < 1e-3


def _wkv_inputs(H, dk, dv, T=18):
    return rnd(3, T, H * dk), rnd(3, T, H * dk, seed=1), rnd(3, T, H * dv, seed=2), -torch.exp(rnd(3, T, H * dk, seed=3) - 1), rnd(H, dk, seed=4)


def _wkv_wanted(r_, k, v, lw, u, H, dk, dv):
    heads = lambda x, n: [t.view(H, n).to(D64) for t in x]
    return [torch.stack(O.wkv(heads(r_[r], dk), heads(k[r], dk), heads(v[r], dv), heads(lw[r].exp(), dk), u.to(D64))) for r in range(r_.shape[0])]


@pytest.mark.parametrize("H,dk,dv", [(2, 6, 6), (3, 5, 7), (1, 8, 8)])
def test_decay_per_channel_with_a_bonus(H, dk, dv):
    args = _wkv_inputs(H, dk, dv)
    want = _wkv_wanted(*args, H, dk, dv)
    got = recurrence.bonus_decay(*args, H)
    assert all(torch.allclose(got[r].to(D64), want[r], atol=1e-5) for r in range(3))
    for _ in range(2):
        state = 9 * torch.ones(4, H, dk, dv)
        on_schedule(lambda rows, s, e: recurrence.bonus_decay(*(pieces(x, s, e) for x in args[:4]), args[4], H, rows, state), want)
    assert bool((state[1] == 9).all())


@pytest.mark.parametrize("window", [1, 5, 8, 40, None])
@pytest.mark.parametrize("heads", [paged.Heads(4, 2, 8, 5), paged.Heads(3, 1, 6, 9)])
def test_sigmoid_weights_in_a_window(heads, window):
    """Keys sit in shuffled pages; one key at a time stands out for the last query: just inside and just outside its window, and at page borders."""
    T, page = 31, 8
    H, G, dk, dv = heads
    table = torch.tensor([[5, 0, 3, 7], [2, 6, 4, 8]], dtype=torch.int32)
    gain, bias, cap = 1 + 0.1 * rnd(H, seed=5), 0.3 * rnd(H, seed=6) - 7, 30.0
    lo = 0 if window is None else max(T - window, 0)
    for target in sorted({0, 7, 8, T - 1, lo, max(lo - 1, 0)}):
        qkv = rnd(2, T, heads.packed, seed=target)
        q, k = qkv[..., :H * dk], qkv[..., H * dk:(H + G) * dk]
        k[0, target] = 12 * torch.nn.functional.normalize(k[0, target].view(G, dk), dim=-1).reshape(-1)
        q[0, -1] = k[0, target].view(G, dk).repeat_interleave(H // G, 0).reshape(-1) / 4
        pos = torch.arange(T, dtype=torch.int32)[None].repeat(2, 1)
        pages = paged.Pages(*(torch.full((10, page, G, max(dk, dv)), 99.0) for _ in range(2)), table, page, None)
        packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
        visible = paged.Visible(window=window, softcap=cap, gain=gain, sigmoid=bias)
        got = paged.paged_attend(packed[:, :, :H], heads, pos, pages, 0.5, visible=visible)
        one = paged.paged_attend(packed[:, -1:, :H], heads, pos[:, -1:].contiguous(), pages, 0.5, visible=visible)
        for r in range(2):
            split = [qkv[r, t].to(D64).split([H * dk, G * dk, G * dv]) for t in range(T)]
            qs, ks, vs = ([s[j].view(n, d) for s in split] for j, (n, d) in enumerate(((H, dk), (G, dk), (G, dv))))
            want = torch.stack(O.sigmoid_attend(qs, ks, vs, 0.5, gain.to(D64), bias.to(D64), cap, window))
            assert torch.allclose(got[r].to(D64), want, atol=1e-4) and torch.allclose(one[r, 0].to(D64), want[-1], atol=1e-4)
        v = qkv[0, target, (H + G) * dk:].view(G, dv).repeat_interleave(H // G, 0)
        assert torch.allclose(got[0, -1], v, atol=0.35) == (target in O.in_window(T - 1, window))      # it came in whole, or is out of sight


def test_weights_are_not_shared_out():
    """Twice the same token: a softmax would give each half the weight; here both count in full."""
    heads = paged.Heads(1, 1, 4, 3)
    qkv = rnd(1, 1, heads.packed).repeat(1, 5, 1)
    pages = paged.Pages(*(torch.zeros(2, 8, 1, 4) for _ in range(2)), torch.zeros(1, 1, dtype=torch.int32), 8, None)
    pos = torch.arange(5, dtype=torch.int32)[None]
    packed = paged.qk_norm_append(qkv, heads, None, None, 0.0, None, pos, pages)
    got = paged.paged_attend(packed[:, :, :1], heads, pos, pages, 0.5, visible=paged.Visible(sigmoid=torch.zeros(1)))
    assert torch.allclose(got[0, :, 0], got[0, 0, 0] * torch.arange(1, 6)[:, None], atol=1e-5)


def test_norm_of_one_number_two_branches_and_what_joins():
    T, d = 4, 10
    H, y, y2, w = rnd(T, 1, d, seed=1), rnd(T, d, seed=2), rnd(T, d, seed=3), torch.tensor(0.7)
    table, add, tokens = rnd(9, d, seed=4), rnd(d, seed=5), torch.tensor([3, 0, 8, 3])
    for write in (None, streams.Write(y, gain=0.8, y2=y2, gain2=0.5), streams.Write(y)):
        for join in (None, streams.Join(add), streams.Join(add, table, tokens), streams.Join(None, table, tokens, 2.0)):
            got, H2 = streams.stream_step(H.clone(), write, None, w, 0.2, torch.float32, "rms", 0.0, join)
            for t in range(T):
                new = H[t, 0].to(D64)
                if write is not None:
                    new = new + (0.8 * y[t] + 0.5 * y2[t] if write.y2 is not None else y[t])
                if join is not None:
                    new = new + (0 if join.add is None else add) + (0 if join.table is None else join.gain * table[tokens[t]])
                assert torch.allclose(H2[t, 0].to(D64), new, atol=1e-6)
                assert torch.allclose(got[t].to(D64), O.scalar_norm(new, w.to(D64), 0.2), atol=1e-5)
    with pytest.raises(NotImplementedError):
        streams.stream_step(rnd(T, 2, d), None, None, w, 0.2, torch.float32, "rms", 0.0, streams.Join(add))


@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (8, 3, 4, 2), (5, 2, 1, 1), (12, 4, 2, 1)])
def test_groups_count_their_best_expert(E, top, groups, keep):
    z = 2 * rnd(60, E)
    z[0] -= 200
    z[1, :2], z[1, 2:] = torch.tensor([5.0, -9.0]), torch.linspace(4.5, 4.0, E - 2)    # a lone best expert beside groups of two good ones
    s = moe_serve.Selection(E, top, groups, keep, float("-inf"), "softmax", False, 1.7, 1)
    w, ids, _ = moe_serve.select_reference(z, None, s)
    for t in range(60):
        chosen, weights = O.route(z[t].to(D64), top, groups, keep, 1.7)
        assert sorted(ids[t].tolist()) == sorted(chosen)
        assert torch.allclose(w[t][ids[t].argsort()].to(D64), weights[torch.tensor(chosen).argsort()], atol=1e-6)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_matches_the_restated_decoder(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name)
    n = 70 if name != "wide" else 40
    tokens, want, layers = C.wanted(name, n)
    got = m(torch.tensor([tokens]))[0]
    assert C.error(got, want) < TOL
    seen = []
    m._static(torch.tensor([tokens]), None, None, observe=lambda r, total: seen.append(total[0].clone()))
    assert len(seen) == len(layers)
    for a, b in zip(seen, layers):
        assert torch.allclose(a.to(D64), b, atol=1e-4 * float(b.abs().max()))
    for size in (1, 2, 3, 16, 33, n):
        assert C.error(C.replay(m, C.cut(tokens, size)), want) < TOL, size
    assert C.error(C.replay(m, [tokens[:n - 20]] + C.cut(tokens[n - 20:], 1)), want) < TOL


PARTS = ["left.q.b", "left.k.b", "left.v.b", "left.q.conv", "left.k.conv", "left.v.conv", "left.temp", "left.pb", "left.o.b", "right.mu.r", "right.mu.k", "right.mu.v",
         "right.mu.g", "right.mu.w", "right.r", "right.k", "right.v", "right.g", "right.w1", "right.w2", "right.w0", "right.u", "right.norm"]
PARTS = ["l0.mix." + p for p in PARTS] + ["l1.mix." + p for p in ("q", "k", "v", "g", "i", "f", "i.b", "f.b", "norm")] + \
    ["l2.mix." + p for p in ("q", "k", "v", "g", "b", "a", "A_log", "dt_bias", "norm", "q.conv", "k.conv", "v.conv")] + \
    ["l0.norm1", "l0.norm2", "final.norm", "loop.step", "l0.mlp.router", "l1.mlp.e1.down", "l0.mlp.e2.gate"]


@pytest.mark.parametrize("part", PARTS)
def test_every_tensor_moves_the_logits(tmp_path, part):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    moved = w[part].float().roll(1, 0) * 1.5 if w[part].dim() else w[part].float() * 1.5
    other = {**w, part: moved.to(torch.bfloat16)}
    tokens = C.prompt(cfg, 24)
    b = Pretrained.load(C.write(tmp_path / "b", cfg, other), dtype=torch.float32)
    want = O.run(cfg, other, tokens)[0]
    with torch.no_grad():
        assert C.error(C.replay(b, [tokens]), want) < TOL
    assert C.error(C.wanted("plain", 24)[1], want) > 3e-3


LEFT = lambda c: c["layers"][0]["mixer"]["left"]
CHANGES = {"window one longer": lambda c: LEFT(c)["mask"].update(size=8), "window one shorter": lambda c: LEFT(c)["mask"].update(size=6),
           "cap": lambda c: LEFT(c).update(softcap=2.0), "scale": lambda c: LEFT(c).update(scale=0.45), "base": lambda c: LEFT(c)["rot"].update(base=200.0),
           "turned part": lambda c: LEFT(c)["rot"].update(dims=6), "left scale": lambda c: c["layers"][0]["mixer"].update(left_scale=0.8),
           "right scale": lambda c: c["layers"][0]["mixer"].update(right_scale=0.7), "gate cap": lambda c: c["layers"][1]["mixer"].update(gate_cap=3.0),
           "eps": lambda c: c["norm"].update(eps=0.05), "experts chosen": lambda c: c["layers"][0]["mlp"]["router"].update(top=3),
           "groups kept": lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1), "groups": lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=2, keep=1),
           "router scale": lambda c: c["layers"][0]["mlp"]["router"].update(scale=1.0), "loop start": lambda c: c["loop"].update(start=1),
           "loop stop": lambda c: c["loop"].update(stop=3), "passes": lambda c: c["loop"].update(times=1)}


@pytest.mark.parametrize("change", sorted(CHANGES))
def test_every_constant_is_read(tmp_path, change):
    cfg = copy.deepcopy(C.CASES["plain"])
    CHANGES[change](cfg)
    w, tokens = C.tensors(C.CASES["plain"]), C.prompt(cfg, 40)
    if "loop" in cfg:
        w["loop.step"] = w["loop.step"][:cfg["loop"]["times"]]
    m = Pretrained.load(C.write(tmp_path / "m", cfg, w), dtype=torch.float32).eval()
    want = O.run(cfg, w, tokens)[0]
    with torch.no_grad():
        assert C.error(m(torch.tensor([tokens]))[0], want) < TOL
        assert C.error(C.replay(m, [tokens[:20]] + C.cut(tokens[20:], 1)), want) < TOL
    assert C.error(C.wanted("plain", 40)[1], want) > 1e-3


def test_nothing_past_the_window_and_the_taps_reaches_a_token(tmp_path):
    cfg, w, m = C.load(tmp_path, "sealed")                                # a window of six behind three taps
    tokens = C.prompt(cfg, 29)
    moved_one = tokens[:11] + [(tokens[11] + 1) % cfg["vocab"]] + tokens[12:]
    for parts in (lambda t: [t], lambda t: C.cut(t, 5), lambda t: [t[:12]] + C.cut(t[12:], 1), lambda t: C.cut(t, 2)):
        diff = (C.replay(m, parts(moved_one)) - C.replay(m, parts(tokens))).abs().amax(-1)
        assert float(diff[:11].max()) == 0 and bool((diff[11:19] > 1e-3).all()) and float(diff[19:].max()) < 1e-5


@pytest.mark.parametrize("name", ["odd", "plain", "looped"])
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
    cfg, w, m = C.load(tmp_path, "looped")
    tokens, want, _ = C.wanted("looped", 180)
    assert C.error(C.replay(m, [tokens[:3]] + C.cut(tokens[3:], 1)), want) < TOL


def test_what_a_layer_keeps(tmp_path):
    cfg, w, m = C.load(tmp_path, "plain")
    slots = m.cache_slots()
    assert len(slots) == 5 and slots[0].beside.state == (3, 5, 5) and dict(slots[0].more) == {"conv": (32 + 16 + 24, 2)} and dict(slots[1].more) == {"n": (2, 7), "m": (2,)}
    store = KVStore(KVCache(page_size=8), 5, 2, 32, 0, 0, torch.float32, "cpu", slots=slots)
    assert store.beside == {0: 5, 2: 6} and store.layer_runs == 5 and store.keeps_state and len(store.slots) == 7
    assert store.k[0] is not None and store.k[5] is None and store.states[5].shape == (2, 3, 5, 5)
    assert len(store.kept_states()) == 2 + 2 * 2 + 2 * 3 + 2              # taps, time mixers (state, token), memories (state, n, m), the delta layer
    assert CacheSlot(more=(("conv", (3, 1)),)).stateful and not CacheSlot(1, 4, 4).stateful


# ------------------------------------------------------------------------------------------------ generation
def _greedy(cfg, w, tokens, n):
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(O.run(cfg, w, seq)[0][-1].argmax()))
    return seq[len(tokens):]


def test_greedy_generation_through_generate_and_the_server(tmp_path):
    from dew_b200.inference import Server
    cfg, w, m = C.load(tmp_path, "plain")
    prompts = [C.prompt(cfg, n, seed=n) for n in (1, 9, 26)]
    want = [_greedy(cfg, w, p, 5) for p in prompts]
    gen = generate(m, None, prompts, 5, sampling=Sampling(temperature=0.0))
    assert [gen.new_tokens(r).tolist() for r in range(3)] == want
    server = Server(m, slots=2, capacity=64, kv_cache=KVCache(page_size=8), chunk=7)       # prompts in portions, slots and pages re-used
    assert server(prompts + prompts[::-1], max_new_tokens=5) == want + want[::-1]
    assert server.ledger.available() == server.ledger.pages
    shared = prompts[2][:17] + prompts[1]                             # a prefix another prompt has left in the pool: its states are gone, so it is read anew
    hits = server.ledger.hits
    assert server([shared], max_new_tokens=5) == [_greedy(cfg, w, shared, 5)] and server.ledger.hits == hits


def test_the_stack_trains_in_its_differentiable_form(tmp_path):
    cfg, _, m = C.load(tmp_path, "plain")
    for p in m.parameters():
        p.requires_grad_(True)
    m.train()
    tokens = torch.tensor([C.prompt(cfg, 30), C.prompt(cfg, 30, 2), C.prompt(cfg, 30, 3)])
    loss = torch.nn.functional.cross_entropy(m(tokens[:, :-1]).flatten(0, 1), tokens[:, 1:].flatten())
    loss.backward()
    assert not [n for n, p in m.named_parameters() if p.grad is None or not bool(torch.isfinite(p.grad).all())]
    assert m.pop_aux()["balance_loss"] is not None and m.param_count(active=True) < m.param_count()


def test_combinations_that_are_not_built_are_refused():
    from dew_b200.models.causal_transformer import CausalTransformer, Loop, TransformerConfig
    base = dict(vocab_size=11, emb_features=8, num_layers=2, num_heads=2, head_dim=4, max_seq_len=32, tie_embeddings=False, qk_norm=False)
    with pytest.raises(NotImplementedError):
        TransformerConfig(**base, norm_one=True)
    with pytest.raises(NotImplementedError):
        TransformerConfig(**base, loop=Loop(2, restate=True))
    with pytest.raises(NotImplementedError):
        Loop(2, step_vectors=True, exit_gate=True)
    with pytest.raises(NotImplementedError):
        CausalTransformer(TransformerConfig(**base, fp32_residual=True, layer_types=("pair",), mixer_options={"left": ("attention", {}), "right": ("nope", {})}))
    for bad in (dict(attn_weighting="relu"), dict(attn_weighting="sigmoid", attention_sinks=True)):
        with pytest.raises(ValueError):
            CausalTransformer(TransformerConfig(**base, fp32_residual=True, layer_types=("nope",), **bad))


# ------------------------------------------------------------------------------------------------ release format
@pytest.mark.parametrize("name", ["odd", "plain", "looped"])
def test_release_round_trip(tmp_path, name):
    cfg, w, m = C.load(tmp_path, name, torch.bfloat16)
    Pretrained.save(m, tmp_path / "again")
    assert json.loads((tmp_path / "again" / "config.json").read_text()) == cfg
    from dew_b200.interop.release import Release
    stored = Release(tmp_path / "again")
    assert set(stored) == set(w) and all(torch.equal(stored[k].float(), w[k].float()) for k in w)
    tokens = torch.tensor([C.prompt(cfg, 12)])
    assert torch.equal(Pretrained.load(tmp_path / "again", dtype=torch.float32)(tokens), Pretrained.load(tmp_path / "model", dtype=torch.float32)(tokens))


def test_defaults_of_a_release(tmp_path):
    """Keys that may be left out: value widths and key heads that equal the others, groups and the router's factor, an empty loop."""
    cfg = copy.deepcopy(C.CASES["once"])
    w = C.tensors(cfg, "once")
    tokens = C.prompt(cfg, 20)
    want = O.run(cfg, w, tokens)[0]
    short = copy.deepcopy(cfg)
    for layer in short["layers"]:
        layer["mixer"].pop("vdim")
        layer["mixer"].pop("kv_heads", None)
        if layer["mlp"]:
            layer["mlp"]["router"].pop("groups")
            layer["mlp"]["router"].pop("scale")
        else:
            layer.pop("mlp")
    m = Pretrained.load(C.write(tmp_path / "a", short, w), dtype=torch.float32)
    with torch.no_grad():
        assert C.error(m(torch.tensor([tokens]))[0], want) < TOL
        short["loop"] = {"start": 1, "stop": 1, "times": 1}
        m = Pretrained.load(C.write(tmp_path / "b", short, w), dtype=torch.float32)
        none = {k: v for k, v in cfg.items() if k != "loop"}
        assert C.error(m(torch.tensor([tokens]))[0], O.run(none, w, tokens)[0]) < TOL


def test_releases_that_do_not_fit_are_refused(tmp_path):
    cfg, w = C.CASES["plain"], C.tensors(C.CASES["plain"])
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "a", cfg, {**w, "l1.mix.q.conv": w["l2.mix.q.conv"]}))
    with pytest.raises(KeyError):
        Pretrained.load(C.write(tmp_path / "b", cfg, {k: v for k, v in w.items() if k != "l0.mix.left.temp"}))
    for name in ("l1.mlp.e1.up", "l0.mix.right.w2", "l2.mix.k.conv", "loop.step"):
        with pytest.raises(ValueError):
            Pretrained.load(C.write(tmp_path / "c", cfg, {**w, name: w[name][:1]}))
    for change in (lambda l: l[0].update(type="convolution"), lambda l: l[0]["mlp"].update(kind="dense"), lambda l: l[0]["mixer"]["left"]["rot"].update(dims=9)):
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
    built = lookup("rarelorn", "model")(**cfg)
    assert built.config.kinds() == Pretrained.load(tmp_path / "model").config.kinds() == ["pair", "mlstm", "gdn"] and built.family == "rarelorn"


def test_trace_run_replays_a_batch(tmp_path):
    cfg, w, _ = C.load(tmp_path, "looped")
    (a, wa, _), (c, wc, _) = C.wanted("looped", 30, 5), C.wanted("looped", 12, 6)
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
