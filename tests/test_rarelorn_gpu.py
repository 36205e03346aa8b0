"""The Rarelorn design on a GPU: its kernels against the plain PyTorch forms, whole models in fp32 and bf16 against the restated decoder on every
schedule, and generation through both entry points (the server with its CUDA graph)."""
import pytest
import torch

import rarelorn_cases as C
import rarelorn_oracle as O

from dew_b200.nn.kv_cache import CacheSlot, KVCache, KVStore
from dew_b200.ops import library, moe_serve, paged, recurrence, rotary, streams, token_mix

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]


def rnd(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype).to(DEV)


def close(got, want, rel):
    return got.shape == want.shape and float((got.float() - want.float()).abs().max()) <= rel * float(want.float().abs().max().clamp_min(1e-6))


def fine(dtype, coarse=1e-2, exact=1e-5):
    return exact if dtype == torch.float32 else coarse


# portions of three rows (one rests at times), down to two tokens and one, with rows at one place and at different ones
SCHEDULE = [(130, 64, 1), (132, 64, 3), (196, 65, 67), (197, 66, 68), (198, 66, 69), (300, 300, 260)]


def portions(T=300):
    """(rows, cut): what ``token_mix`` needs of each portion, and a function that cuts ``x [3, T, C]`` to it (padded with noise)."""
    at = (0, 0, 0)
    for nxt in SCHEDULE:
        n = max(e - s for s, e in zip(at, nxt))
        n = n if n == 1 else (n + 127) // 128 * 128
        pos = torch.full((3, n), -1, dtype=torch.int32)
        for r in range(3):
            pos[r, :nxt[r] - at[r]] = torch.arange(at[r], nxt[r])
        rows = token_mix.Rows(pos.to(DEV), (pos.amax(1) + 1).to(torch.int32).to(DEV), torch.tensor([2, 0, 3], dtype=torch.int32, device=DEV))

        def cut(x, at=at, nxt=nxt, n=n):
            out = torch.full((3, n, *x.shape[2:]), 3.0, dtype=x.dtype, device=DEV)
            for r in range(3):
                out[r, :nxt[r] - at[r]] = x[r, at[r]:nxt[r]]
            return out
        yield rows, cut, at, nxt
        at = nxt


def against(call, plain, rel):
    """``call`` and ``plain``: (rows, cut) -> outputs ``[3, n, ...]``, on every portion, each over states of its own."""
    for rows, cut, at, nxt in portions():
        got, want = call(rows, cut), plain(rows, cut)
        for r in range(3):
            n = nxt[r] - at[r]
            assert n == 0 or close(got[r, :n], want[r, :n], rel), (at, nxt, r)
            assert not got[r, n:].any()


# ------------------------------------------------------------------------------------------------ neighbours, norms, small products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C_,taps,wide", [(64, 4, 80), (24, 3, 24), (40, 2, 48), (1030, 4, 1030), (16, 1, 16), (33, 6, 35), (264, 4, 271), (32, 9, 32)])
def test_short_convolution(dtype, C_, taps, wide):
    x, w, b = rnd(3, 300, wide, dtype=dtype), rnd(C_, taps, seed=1, dtype=dtype), rnd(C_, seed=2, dtype=dtype)
    for silu, bias in ((True, None), (False, b)):
        one, two = (torch.full((4, C_, taps - 1), 9.0, device=DEV) for _ in range(2))
        against(lambda rows, cut: token_mix.conv_tokens(cut(x)[..., :C_], w, bias, silu, rows, one),
                lambda rows, cut: token_mix.conv_tokens_reference(cut(x).float()[..., :C_], w, bias, silu, rows, two), fine(dtype))
        assert taps == 1 or close(one, two, 1e-6)
        assert close(token_mix.conv_tokens(x[..., :C_], w, bias, silu), token_mix.conv_tokens_reference(x.float()[..., :C_], w, bias, silu), fine(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,n", [(64, 5), (37, 3), (2056, 1)])
def test_token_shift(dtype, d, n):
    x, mu = rnd(3, 300, d, dtype=dtype), torch.rand(n, d, device=DEV).to(dtype)
    one, two = (torch.full((4, d), 9.0, device=DEV) for _ in range(2))
    against(lambda rows, cut: token_mix.shift_tokens(cut(x), mu, rows, one).permute(1, 2, 0, 3),
            lambda rows, cut: token_mix.shift_tokens_reference(cut(x).float(), mu, rows, two).permute(1, 2, 0, 3), fine(dtype))
    assert torch.equal(one, two)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 70, 600])
def test_small_products_and_gated_norms(dtype, T):
    for d, n in ((64, 8), (37, 3), (4096, 64), (200, 130)):
        x, w = rnd(1, T, d, dtype=dtype), rnd(n, d, seed=1, dtype=dtype)
        assert close(token_mix.narrow_product(x, w).double(), torch.nn.functional.linear(x.double(), w.double()), 1e-5)
    for rank, C_ in ((16, 176), (6, 37), (64, 256), (5, 70), (33, 8)):
        z, w2, w0 = rnd(1, T, rank), rnd(C_, rank, seed=1, dtype=dtype) * rank ** -0.5, rnd(C_, seed=2, dtype=dtype) - 2
        want = -torch.exp(torch.nn.functional.linear(torch.tanh(z.double()), w2.double(), w0.double()))
        assert float(((token_mix.low_rank_decay(z, w2, w0).double() - want) / want).abs().max()) < 1e-4
    for H, d in ((4, 64), (3, 5), (2, 96), (1, 300), (7, 128)):
        x, g = rnd(2, T, H, d, dtype=dtype), rnd(2, T, H * d + 8, seed=1, dtype=dtype)
        for act in ("silu", "sigmoid"):
            for w in (rnd(d, seed=2, dtype=dtype), rnd(H * d, seed=3, dtype=dtype)):
                assert close(token_mix.head_gated_norm(x, g[..., 8:], w, 1e-2, act), token_mix.head_gated_norm_reference(x.float(), g[..., 8:].float(), w, 1e-2, act), fine(dtype))
    x, w = rnd(4, 1, T, 40, dtype=dtype), rnd(4, 24, 40, seed=1, dtype=dtype)
    for got, a, b in zip(token_mix.own_products(x, w), x, w):
        assert close(got, torch.nn.functional.linear(a.float(), b.float()), fine(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [64, 4096, 1100, 7, 9000])
def test_residual_step_with_a_norm_of_one_number(dtype, d):
    T = 9
    H, y, y2, w = rnd(T, 1, d, seed=2), rnd(T, d, seed=3, dtype=dtype), rnd(T, d, seed=4, dtype=dtype), torch.tensor(0.7, dtype=dtype, device=DEV)
    table, add, tokens = rnd(50, d, seed=5, dtype=dtype), rnd(d, seed=6, dtype=dtype), torch.randint(0, 50, (T,), device=DEV)
    for write in (None, streams.Write(y), streams.Write(y, gain=0.8, y2=y2, gain2=0.5), streams.Write(y, add, y2=y2, scale2=add, gain=2.0)):
        for join in (None, streams.Join(add), streams.Join(add, table, tokens), streams.Join(None, table, tokens, 2.0)):
            ref, H_ref = streams.stream_step_reference(H, write, None, w, 1e-2, dtype, "rms", 0.0, join)
            got, H_got = streams.stream_step(H.clone(), write, None, w, 1e-2, dtype, "rms", 0.0, join)
            assert close(H_got, H_ref, 1e-5) and close(got, ref, fine(dtype))


# ------------------------------------------------------------------------------------------------ recurrences
SIZES = [(4, 2, 64, 64), (3, 3, 32, 48), (2, 1, 128, 128), (2, 2, 96, 72), (3, 1, 8, 136), (2, 2, 5, 7), (2, 2, 20, 33), (1, 1, 200, 40), (1, 1, 300, 9),
         (26, 13, 64, 72), (25, 25, 128, 128)]        # (the last two: enough heads for the wide blocks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv", SIZES)
def test_gated_delta_rule(dtype, H, G, dk, dv):
    z = rnd(3, 300, 2 * G * dk + H * dv, dtype=dtype)
    gates, A, dt = 2 * rnd(3, 300, 2 * H, seed=1), rnd(H, seed=2) - 1, rnd(H, seed=3)
    split = lambda x: x.split([G * dk, G * dk, H * dv], -1)
    for kernel in [None] + (["sequence"] if dtype == torch.bfloat16 else []):
        one, two = (torch.full((4, H, dk, dv), 9.0, device=DEV) for _ in range(2))
        against(lambda rows, cut: recurrence.delta_rule(*split(cut(z)), cut(gates), A, dt, H, G, None, rows, one, kernel),
                lambda rows, cut: recurrence.delta_rule_reference(*split(cut(z).float()), cut(gates), A, dt, H, G, dk ** -0.5, rows, two), fine(dtype, exact=3e-5))
        assert close(one, two, 1e-4) and bool((one[1] == 9).all())
    got = recurrence.delta_rule(*split(z), gates, A, dt, H, G)
    assert close(got, recurrence.delta_rule_reference(*split(z.float()), gates, A, dt, H, G, dk ** -0.5), fine(dtype, exact=3e-5))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", sorted({(H, dk, dv) for H, _, dk, dv in SIZES}))
def test_matrix_memory(dtype, H, dk, dv):
    z = rnd(3, 300, 2 * H * dk + 2 * H * dv, dtype=dtype)
    gates, bi, bf = 3 * rnd(3, 300, 2 * H, seed=1), rnd(H, seed=2), rnd(H, seed=3) + 1
    split = lambda x: x.split([H * dk, H * dk, H * dv, H * dv], -1)[:3]
    fresh = lambda: recurrence.Memory(*(torch.full(s, 9.0, device=DEV) for s in ((4, H, dk, dv), (4, H, dk), (4, H))))
    for kernel in [None] + (["sequence"] if dtype == torch.bfloat16 else []):
        for cap in (15.0, 2.0):
            one, two = fresh(), fresh()
            against(lambda rows, cut: recurrence.matrix_memory(*split(cut(z)), cut(gates), bi, bf, H, cap, None, rows, one, kernel),
                    lambda rows, cut: recurrence.matrix_memory_reference(*split(cut(z).float()), cut(gates), bi, bf, H, cap, dk ** -0.5, rows, two),
                    fine(dtype, exact=2e-4))
            assert all(close(a, b, 1e-3) for a, b in zip(one, two)) and bool((one.m[1] == 9).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", sorted({(H, dk, dv) for H, _, dk, dv in SIZES}))
def test_decay_per_channel(dtype, H, dk, dv):
    r, k, v, u = rnd(3, 300, H * dk, dtype=dtype), rnd(3, 300, H * dk, seed=1, dtype=dtype), rnd(3, 300, H * dv, seed=2, dtype=dtype), rnd(H, dk, seed=3, dtype=dtype)
    for shift in (-1.0, -4.0, 3.0):                                     # also channels that forget everything at every token
        lw = -torch.exp(1.5 * rnd(3, 300, H * dk, seed=4) + shift)
        for kernel in [None] + (["sequence"] if dtype == torch.bfloat16 else []):
            one, two = (torch.full((4, H, dk, dv), 9.0, device=DEV) for _ in range(2))
            against(lambda rows, cut: recurrence.bonus_decay(cut(r), cut(k), cut(v), -cut(-lw).abs(), u, H, rows, one, kernel),
                    lambda rows, cut: recurrence.bonus_decay_reference(cut(r).float(), cut(k).float(), cut(v).float(), -cut(-lw).abs(), u, H, rows, two),
                    fine(dtype, exact=3e-5))
            assert close(one, two, 1e-4) and bool((one[1] == 9).all())


def test_gates_at_their_ends():
    """Steps of 0 and 1, decays of 0 and 1, input gates that raise the maximum by thirty at once, and a long stretch that forgets nothing."""
    H, d, T = 2, 64, 200
    z = rnd(1, T, 3 * H * d, dtype=torch.bfloat16)
    q, k, v = z.split(H * d, -1)
    gates = torch.zeros(1, T, 2 * H, device=DEV)
    gates[:, ::3, :H], gates[:, 1::3, :H] = 40.0, -40.0
    gates[:, :100, H:], gates[:, 100, H:] = -60.0, 60.0
    A, dt = torch.full((H,), 3.0, device=DEV), torch.zeros(H, device=DEV)
    want = recurrence.delta_rule_reference(q.float(), k.float(), v.float(), gates, A, dt, H, H, d ** -0.5)
    assert close(recurrence.delta_rule(q, k, v, gates, A, dt, H, H), want, 1e-2) and close(recurrence.delta_rule(q, k, v, gates, A, dt, H, H, kernel="sequence"), want, 1e-2)
    gates = torch.full((1, T, 2 * H), -60.0, device=DEV)
    gates[:, 70::40, :H], gates[:, :, H:] = 60.0, 60.0
    gates[:, 150, H:] = -60.0
    want = recurrence.matrix_memory_reference(q.float(), k.float(), v.float(), gates, dt, dt, H, 15.0, d ** -0.5)
    for kernel in ("chunks", "sequence"):
        got = recurrence.matrix_memory(q, k, v, gates, dt, dt, H, 15.0, kernel=kernel)
        assert bool(torch.isfinite(got).all())
        for a, b in ((0, 70), (70, 151), (151, T)):                     # (the parts differ by orders of magnitude)
            assert close(got[:, a:b], want[:, a:b], 2e-2), (kernel, a)


def test_a_far_write_is_read_back():
    """One key among hundreds that stands out, across chunks of the tensor-core form and into decoding."""
    H, d, T = 2, 64, 400
    z = 0.02 * rnd(1, T, 3 * H * d, dtype=torch.float32)
    mark = torch.nn.functional.normalize(rnd(H, d, seed=5), dim=-1)
    z[0, 37].view(3, H, d)[1] = 4 * mark                                # the key and its value
    z[0, 37].view(3, H, d)[2] = rnd(H, d, seed=6)
    for t in (38, 63, 64, 255, 398, 399):
        z[0, t].view(3, H, d)[0] = mark
    z = z.bfloat16()
    q, k, v = z.split(H * d, -1)
    value = v[0, 37].view(H, d).float()
    rows = token_mix.whole(1, T - 1, DEV)
    last = token_mix.Rows(torch.full((1, 1), T - 1, dtype=torch.int32, device=DEV), torch.full((1,), T, dtype=torch.int32, device=DEV))
    gates = torch.cat([torch.full((1, T, H), -9.0, device=DEV), torch.full((1, T, H), -30.0, device=DEV)], -1)
    gates[:, 37, :H] = 30.0
    st = torch.zeros(1, H, d, d, device=DEV)
    zero = torch.zeros(H, device=DEV)
    cut = lambda a, b: (q[:, a:b], k[:, a:b], v[:, a:b], gates[:, a:b])
    got = torch.cat([recurrence.delta_rule(*cut(0, T - 1), zero, zero, H, H, 1.0, rows, st), recurrence.delta_rule(*cut(T - 1, T), zero, zero, H, H, 1.0, last, st)], 1)
    for t in (38, 63, 64, 255, 398, 399):
        assert close(got[0, t], value, 2e-2), t
    assert float(got[0, 36].abs().max()) < 0.05 * float(value.abs().max())


def test_the_chunked_form_refuses_what_it_cannot_take():
    with pytest.raises(ValueError):
        recurrence.bonus_decay(*(rnd(1, 4, 10, dtype=torch.bfloat16) for _ in range(3)), -rnd(1, 4, 10).abs(), rnd(2, 5), 2, kernel="chunks")


# ------------------------------------------------------------------------------------------------ attention
HEADS = [(paged.Heads(5, 1, 96, 88), 96), (paged.Heads(8, 2, 64, 64), 32), (paged.Heads(6, 2, 128, 80), 64), (paged.Heads(12, 1, 24, 40), 24),
         (paged.Heads(2, 2, 200, 130), 8), (paged.Heads(3, 1, 7, 5), 4), (paged.Heads(4, 4, 128, 128), 128), (paged.Heads(6, 3, 72, 160), 40)]


@pytest.mark.parametrize("S,D,Hq,Hkv,window,cap", [(512, 128, 4, 2, 96, 20.0), (512, 64, 4, 1, 128, 0.0), (640, 64, 2, 2, 300, 5.0), (384, 128, 3, 1, 1, 0.0),
                                                  (1280, 128, 2, 1, None, 30.0), (1280, 64, 2, 1, 129, 2.0)])
def test_flash_forward_with_sigmoid_weights(S, D, Hq, Hkv, window, cap):
    from dew_b200.nn.kv_cache import visible_attention
    from dew_b200.ops.flash import Variants, flash_fwd
    q, k, v = (rnd(2, S, h, D, seed=i, dtype=torch.bfloat16) for i, h in enumerate((Hq, Hkv, Hkv)))
    gain, bias = 0.5 + torch.rand(Hq, device=DEV), rnd(Hq, seed=5) - 3
    got, _ = flash_fwd(q, k, v, True, 0.3, need_lse=False, var=Variants(window, cap, gain=gain, sigmoid=bias))
    want = visible_attention(q.float(), k.float(), v.float(), 0.3, paged.Visible(None, None, window, 0, cap, gain, bias))
    assert close(got, want, 1.5e-2)
    got, _ = flash_fwd(q, k, v, True, 0.3, need_lse=False, var=Variants(window, cap, gain=gain))                # the factors alone, under a softmax
    assert close(got, visible_attention(q.float(), k.float(), v.float(), 0.3, paged.Visible(None, None, window, 0, cap, gain)), 1.5e-2)
    library.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 48, 64, 100, 129, 257, None])
@pytest.mark.parametrize("heads,dims", HEADS)
def test_attention_from_the_packed_projection(dtype, heads, dims, window):
    """``attend_slot``: a prompt, portions at mixed positions, and decode steps, with planted keys just inside and just outside the window and at page
    borders; sigmoid weights, and the softmax with factors."""
    rel = 2e-5 if dtype == torch.float32 else 5e-2
    H, G, dk, dv = heads
    rows, first, T = 3, 128, 300
    rot = rotary.Rotary(dims, 100.0)
    slots = [CacheSlot(G, dk, dv)]
    x = rnd(rows, T, heads.row, seed=3, dtype=dtype)
    back = lambda t, target, at: rotary.turn(rotary.turn(t[None], rotary.angles_reference(torch.tensor([target]), rot), rot) * 1.0,
                                             rotary.angles_reference(torch.tensor([at]), rot) * torch.tensor([1.0, -1.0]), rot)[0]
    k = x[..., H * dk:(H + G) * dk].cpu()
    for at in range(130, T, 13):
        lo = 0 if window is None else max(at - window + 1, 0)
        for r, target in enumerate((lo, max(lo - 1, 0), min(at, at // 64 * 64))):
            q = back(k[r, target].view(G, dk).float(), target, at).repeat_interleave(H // G, 0)
            x[r, at, :H * dk] = (2 * q.reshape(-1)).to(dtype).to(DEV)
    for sigmoid in (True, False):
        kw = dict(scale=dk ** -0.5, eps=1e-3, window=window, softcap=9.0, rot=rot, gain=0.5 + torch.rand(H, generator=torch.Generator().manual_seed(1)).to(dtype).to(DEV),
                  sigmoid=rnd(H, seed=5, dtype=dtype) - 4 if sigmoid else None)
        store = KVStore(KVCache(page_size=64, pages=24), 1, rows, 320, 0, 0, dtype, DEV, slots=slots)
        store.page_table.copy_(torch.randperm(24, generator=torch.Generator().manual_seed(0))[:15].reshape(3, 5).to(DEV))
        cpu = KVStore(KVCache(page_size=64, pages=24), 1, rows, 320, 0, 0, torch.float32, "cpu", slots=slots)
        cpu.page_table.copy_(store.page_table.cpu())
        ckw = {n: v.float().cpu() if isinstance(v, torch.Tensor) else v for n, v in kw.items()}

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
                assert m == 0 or close(got[r, :m].cpu(), want[r, :m], rel), (starts, b, r, sigmoid)
                assert bool(torch.isfinite(got[r]).all())

        at = [first, 77, 1]
        both(at, [0, 0, 0])
        for nxt in ([first + 2, 77 + 61, 1], [199, 199, 130]):
            both(nxt, at)
            at = nxt
        for t in range(0, 101, 1 if sigmoid else 4):
            nxt = [min(at[0] + 1, T), at[1] + (t % 3 > 0), at[2] + 1]
            both(nxt, at)
            at = nxt
    library.check_status()


@pytest.mark.parametrize("D,Hq,Hkv", [(128, 8, 2), (128, 16, 1), (64, 8, 2), (256, 4, 2), (128, 3, 3)])
def test_decode_with_sigmoid_weights_over_long_rows(D, Hq, Hkv):
    heads = paged.Heads(Hq, Hkv, D, D)
    lens = [1, 64, 130, 1000, 1001, 2000, 2001, 2999, 4000, 4064]
    store = KVStore(KVCache(page_size=64), 1, len(lens), 4096, 0, 0, torch.bfloat16, DEV, slots=[CacheSlot(Hkv, D, D)])
    store.k[0].copy_(rnd(*store.k[0].shape, seed=1)), store.v[0].copy_(rnd(*store.v[0].shape, seed=2))
    gain, bias = 0.5 + torch.rand(Hq, device=DEV), rnd(Hq, seed=6) - 2
    for window, cap in ((1000, 20.0), (512, 0.0), (96, 4.0), (None, 20.0), (1, 0.0)):
        qkv, pos = rnd(len(lens), 1, heads.packed, seed=3, dtype=torch.bfloat16), torch.tensor(lens, device=DEV)[:, None] - 1
        pages = paged.Pages(store.k[0].float(), store.v[0].float(), store.page_table, 64, None)
        for sig in (bias, None):
            got = store.attend_slot(0, qkv, heads, pos, scale=0.2, window=window, softcap=cap, gain=gain, sigmoid=sig)
            pages = paged.Pages(store.k[0].float(), store.v[0].float(), store.page_table, 64, None)
            want = paged.paged_attend_reference(qkv[..., :Hq * D].view(len(lens), 1, Hq, D).float(), heads, pos.int(), pages, 0.2,
                                                paged.Visible(None, None, window, 0, cap, gain, sig))
            assert close(got, want, 1.5e-2), (window, cap, sig is None)
    library.check_status()


# ------------------------------------------------------------------------------------------------ the router
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,d,E,top,groups,keep", [(1, 64, 8, 2, 4, 2), (37, 72, 6, 1, 3, 1), (70, 30, 6, 6, 1, 1), (600, 64, 200, 8, 8, 3), (700, 128, 64, 8, 8, 4)])
def test_groups_by_their_best_expert(dtype, T, d, E, top, groups, keep):
    s = moe_serve.Selection(E, top, groups, keep, float("-inf"), "softmax", False, 1.7, 1)
    x, weight = rnd(T, d, dtype=dtype), (2 * d ** -0.5 * rnd(E, d, seed=2)).to(torch.bfloat16).float()
    split = moe_serve.split_weights(weight)
    logits = (x.double() @ weight.double().t()).cpu()
    scores = torch.softmax(logits, -1)
    best = scores.view(T, groups, -1).amax(-1)
    cut = best.topk(keep, -1).values[:, -1:]
    for form in ["rows"] + (["product"] if dtype == torch.bfloat16 and d % 8 == 0 else []):
        r = moe_serve.route(x, weight, split if dtype == torch.bfloat16 else None, None, s, None, kernel=form)
        ids = r.ids.cpu().long()
        assert bool((best.gather(1, ids // (E // groups)) >= cut * (1 - 1e-3)).all()) and all(len(set(row)) == top for row in ids.tolist())
        open_ = scores.view(T, groups, -1).masked_fill((best < cut).unsqueeze(-1), 0.0).view(T, E)
        assert bool((scores.gather(1, ids) >= open_.topk(top, -1).values[:, -1:] * (1 - 1e-3)).all())
        assert close(r.weights.cpu().double(), 1.7 * scores.gather(1, ids), 1e-4)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_model_on_every_schedule(tmp_path, name):
    """fp32, every position."""
    cfg, w, m = C.load(tmp_path, name, torch.float32, DEV)
    tokens, want, _ = C.wanted(name, 150 if name != "wide" else 140)
    good = lambda got, ref=want: C.error(got, ref) < 2e-4
    assert good(C.replay(m, [tokens]))
    for size in (2, 50, 64, 65):
        assert good(C.replay(m, C.cut(tokens, size), pool_tokens=160)), size
    assert good(C.replay(m, [tokens[:100]] + C.cut(tokens[100:], 1)))
    with torch.no_grad():
        assert good(m(torch.tensor([tokens], device=DEV))[0])


def tolerance(tmp_path, name, want, tokens):
    """What rounding alone costs the plain PyTorch forms in bf16 on the CPU, times three; every expert is chosen, so no close call adds to it."""
    _, _, m = C.load(tmp_path / "cpu", name, torch.bfloat16, sure=True)
    return 3 * C.error(C.replay(m, [tokens]), want)


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_bf16_model_on_every_schedule(tmp_path, name):
    """Every position of prompts, portions and decode steps, and a batch of unequal rows on re-used rows and pages."""
    tokens, want, _ = C.wanted(name, 150 if name != "wide" else 140, sure=True)
    tol = tolerance(tmp_path, name, want, tokens)
    assert tol < 0.5
    cfg, w, m = C.load(tmp_path, name, torch.bfloat16, DEV, sure=True)
    good = lambda got, ref=want: C.error(got, ref) < tol
    assert good(C.replay(m, [tokens]))
    for size in (2, 50, 64, 65):
        assert good(C.replay(m, C.cut(tokens, size), pool_tokens=160)), size
    assert good(C.replay(m, [tokens[:60]] + C.cut(tokens[60:], 1)))
    from dew_b200.sampling.text import RowBatch
    lengths = (1, 120, 40)
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
    """bf16 decoding across window, page and chunk borders against the same positions of one prompt."""
    cfg, w, m = C.load(tmp_path, "wide", torch.bfloat16, DEV, sure=True)
    tokens = C.prompt(cfg, 420)
    whole, steps = C.replay(m, [tokens]), C.replay(m, [tokens[:90]] + C.cut(tokens[90:], 1))
    portions_ = C.replay(m, C.cut(tokens, 128))
    assert C.error(steps, whole.cpu()) < 0.2 and C.error(portions_, whole.cpu()) < 0.2


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
    """Rows whose positions change between replays, in bf16; the graph's warm-up must not move a state."""
    from dew_b200.inference import Server
    cfg, w, m = C.load(tmp_path, "wide", torch.bfloat16, DEV)
    prompts = [C.prompt(cfg, n, seed=n) for n in (5, 90, 129)]
    runs = [Server(m, slots=4, capacity=256, kv_cache=KVCache(page_size=page), cuda_graph=g)(prompts, max_new_tokens=12) for g in (False, True)]
    assert runs[0] == runs[1]
