"""The kernels that the Tupunex layers add or extend, alone against the plain functions: several streams mixed with a sublayer's
result and normed as their weighted sum, the rows of differential attention (biases, convolution over portions and slots,
layout and pages), two maps on the attention kernels (one key made to tower just inside or just outside the window, in either
map), and the difference of the maps with its norm and gate.  (The latent rows and the linear per head with a gate per
head: test_tutezen_kernels_gpu.py.)"""
import math

import pytest
import torch

import kernel_utils as K
import plain_tupunex as PX
from atoma_infer_b200.parts.base import PendingSum, StreamMix

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def rts():
    from atoma_infer_b200.engine.runtime import make_runtime

    return {"bfloat16": make_runtime("bfloat16", "cuda:0"), "float32": make_runtime("float32", "cuda:0")}


def _portions(lens, sizes):
    at, step, steps = [0] * len(lens), 0, []
    while any(a < n for a, n in zip(at, lens)):
        cur = []
        for k, n in enumerate(lens):
            c = min(sizes[(step + 2 * k) % len(sizes)], n - at[k])
            if c > 0:
                cur.append((k, at[k], c))
                at[k] += c
        steps.append(cur)
        step += 1
    return steps


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("H", [72, 131, 512, 1030, 2304, 6000, 9216])
def test_streams_mixed_and_normed(rts, dtype, S, H):
    """One to four weighted terms, a factor, a vector and a scale per channel; the streams in place; chosen rows, which leave
    the streams as they are; the plain sum; nothing pending; no norm."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(S * 10000 + H)
    T = 9
    rnd = lambda *shape: torch.randn(*shape, generator=g)  # noqa: E731
    ctx, rows = K.make_context(rt, [(0, 4), (7, 5)], 16, [[1], [2]], rows=(8, 2, 2))
    x, w, ls, vec = rnd(T, S * H), 1 + 0.2 * rnd(H), rnd(H), rnd(H)
    M, give, read = rnd(S, S), rnd(S), rnd(S)
    ts = [rnd(T, H).to(rt.dtype) for _ in range(3)]
    dev = lambda t: t.to(rt.device) if t is not None else None  # noqa: E731
    tol = 2e-5 if dtype == "float32" else 1e-2
    for terms, fs, mult, v, sc in ((ts[:1], None, 1.0, None, ls), (ts[:1], None, 1.0, None, None), (ts, (0.5, -1.25, 2.0), 0.7, vec, ls)):
        y = torch.zeros(T, H, dtype=torch.float64)
        for t, f in zip(terms, fs or (1.0,) * 3):
            y = y + f * t.double()
        y = mult * y + (v.double() if v is not None else 0)
        y = y * (sc.double() if sc is not None else 1)
        X = PX.mix_streams(x.view(T, S, H).double(), M, give, y)
        pending = StreamMix(PendingSum(tuple(dev(t) for t in terms), mult, vector=dev(v), factors=fs), dev(sc), dev(M), dev(give))
        want = PX.rms_norm(PX.read_streams(X, read), w, 1e-5)
        resid, out = dev(x.clone()), torch.full((T, H), float("nan"), dtype=rt.dtype, device=rt.device)
        rt.ops.stream_mix_norm(resid, S, pending, dev(read), dev(w), 1e-5, out, ctx.meta, T)
        assert torch.allclose(resid.cpu().double(), X.reshape(T, -1), atol=1e-5 * float(X.abs().max()))
        assert torch.allclose(out.float().cpu().double(), want, atol=tol * float(want.abs().max()))
        resid, out = dev(x.clone()), torch.full((3, H), float("nan"), dtype=rt.dtype, device=rt.device)
        rt.ops.stream_mix_norm(resid, S, pending, None, dev(w), 1e-5, out, ctx.meta, 3, rows=rows)
        want = PX.rms_norm(X.sum(1), w, 1e-5)[[8, 2, 2]]
        assert torch.equal(resid.cpu(), x)
        assert torch.allclose(out.float().cpu().double(), want, atol=tol * float(want.abs().max()))
        rt.ops.stream_mix_norm(resid, S, pending, None, None, 0.0, None, ctx.meta, T)
        assert torch.allclose(resid.cpu().double(), X.reshape(T, -1), atol=1e-5 * float(X.abs().max()))
    resid, out = dev(x.clone()), torch.full((T, H), float("nan"), dtype=rt.dtype, device=rt.device)
    rt.ops.stream_mix_norm(resid, S, None, dev(read), dev(w), 1e-5, out, ctx.meta, T)
    want = PX.rms_norm(PX.read_streams(x.view(T, S, H).double(), read), w, 1e-5)
    assert torch.equal(resid.cpu(), x) and torch.allclose(out.float().cpu().double(), want, atol=tol * float(want.abs().max()))
    rt.ops.check_status()


# (heads, key/value heads, maps, map, value, taps): sizes that take 16-byte and 8-byte pieces and single elements
ROWS = [(4, 2, 2, 16, 32, 4), (6, 2, 2, 44, 92, 3), (2, 1, 2, 12, 20, 2), (3, 1, 2, 9, 10, 3), (4, 4, 2, 32, 48, 1), (2, 2, 2, 64, 128, 0),
        (2, 1, 2, 8, 16, 6), (6, 3, 1, 24, 16, 4), (2, 1, 3, 8, 40, 3), (8, 2, 2, 64, 128, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kvh,maps,d,dv,taps", ROWS)
def test_rows_over_portions_and_slots(rts, dtype, heads, kvh, maps, d, dv, taps):
    """Four requests in portions of one to hundreds of tokens in one batch, and decode steps; rings in scattered slots that are
    slices of a wider state and hold another request's rows at the start; NaN wherever nothing may be read from."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(heads * 100 + d)
    page, dp = 8, -(-max(maps * d, dv) // 16) * 16
    n = (heads + kvh) * maps * d + kvh * dv
    lens = [37, 5, 160, 900]
    us = [torch.randn(L, n + heads, generator=g).to(rt.dtype) for L in lens]
    bias, w = torch.randn(n, generator=g), torch.randn(n, max(taps, 1), generator=g)
    want = []
    for u in us:
        r = u[:, :n].double() + bias.double()
        want.append(PX.causal_conv(r, w) if taps else r)
    tables, num_pages = K.scrambled_tables(lens, page, 1)
    slots = [3, 0, 4, 1]
    R = max(taps - 1, 1)
    wide = torch.full((5, 4 + R * n + 4), 7.0, device=rt.device)   # (whatever an earlier request left)
    ring = wide[:, 4:4 + R * n].view(5, R, n) if taps > 1 else None
    cache = torch.full((num_pages, 2, kvh, page, dp), float("nan"), dtype=rt.dtype, device=rt.device)
    dev = lambda t: t.to(rt.device)  # noqa: E731
    tol = 2e-5 if dtype == "float32" else 1.2e-2
    for cur in _portions(lens, (1, 2, 3, 1, 7, 130, 1, 21, 600)):
        ctx, _ = K.make_context(rt, [(a, c) for _, a, c in cur], page, [tables[k] for k, _, _ in cur])
        ctx.state_slots.copy_(torch.tensor([slots[k] for k, _, _ in cur], dtype=torch.int32))
        u = torch.cat([us[k][a:a + c] for k, a, c in cur])
        q = torch.full((ctx.T, heads * maps * dp), float("nan"), dtype=rt.dtype, device=rt.device)
        rt.ops.map_rows(dev(u)[:, :n], ctx, cache, 0, q, heads=heads, kv_heads=kvh, maps=maps, d=d, dv=dv, dp=dp, page_size=page,
                        num_pages=num_pages, store_kv=True, bias=dev(bias), conv_w=dev(w.t().contiguous()) if taps else None, ring=ring)
        ref = torch.cat([want[k][a:a + c] for k, a, c in cur])
        expect = torch.zeros(ctx.T, heads, maps, dp, dtype=torch.float64)
        for m in range(maps):
            expect[:, :, m, m * d:(m + 1) * d] = ref[:, :heads * maps * d].view(ctx.T, heads, maps, d)[:, :, m]
        got = q.float().cpu().double().view(ctx.T, heads, maps, dp)
        assert torch.allclose(got, expect, atol=tol * float(expect.abs().max()))
        assert bool((got[expect == 0] == 0).all())
    rt.ops.check_status()
    for k, L in enumerate(lens):
        pos = torch.arange(L)
        pages = torch.tensor(tables[k])[pos // page]
        got = cache.cpu()[pages, :, :, pos % page].float().double()      # [L, 2, kvh, dp]
        expect = torch.zeros(L, 2, kvh, dp, dtype=torch.float64)
        expect[:, 0, :, :maps * d] = want[k][:, heads * maps * d:(heads + kvh) * maps * d].view(L, kvh, maps * d)
        expect[:, 1, :, :dv] = want[k][:, (heads + kvh) * maps * d:].view(L, kvh, dv)
        assert torch.allclose(got, expect, atol=tol * float(expect.abs().max()))
    if taps > 1:  # the last rows as they were projected, by position; nothing around them
        for k, L in enumerate(lens):
            for p in range(max(L - (taps - 1), 0), L):
                assert torch.equal(ring[slots[k], p % (taps - 1)].cpu(), us[k][p, :n].float())
        assert bool((wide[:, :4] == 7.0).all()) and bool((wide[2] == 7.0).all()) and bool((wide[:, 4 + R * n:] == 7.0).all())


def test_rows_without_a_page_raise_the_status_word(rts):
    rt = rts["float32"]
    ctx, _ = K.make_context(rt, [(0, 3)], 4, [[9]])
    q, cache = torch.zeros(3, 2 * 16, device=rt.device), torch.zeros(4, 2, 1, 4, 16, device=rt.device)
    rt.ops.map_rows(torch.zeros(3, 48, device=rt.device), ctx, cache, 0, q, heads=1, kv_heads=1, maps=2, d=8, dv=16, dp=16, page_size=4,
                    num_pages=4, store_kv=True)
    with pytest.raises(Exception, match="page"):
        rt.ops.check_status()


def _maps_case(rt, entries, heads, kvh, d, dv, page, window, cap, seed, mark=None, fast=True):
    """Two maps of a step's queries over a hand-filled cache, on the attention kernels; the largest difference from the plain
    maps.  ``mark``: (keys, map): per request the key that towers for its last query in that map, if it may be seen."""
    g = torch.Generator().manual_seed(seed)
    dp = -(-max(2 * d, dv) // 16) * 16
    lengths = [c + n for c, n in entries]
    tables, num_pages = K.scrambled_tables(lengths, page, seed)
    qs = [torch.randn(L, heads, 2, d, generator=g) for L in lengths]
    ks, vs = [torch.randn(L, kvh, 2, d, generator=g) for L in lengths], [torch.randn(L, kvh, dv, generator=g) for L in lengths]
    if mark is not None:
        for q, k, key in zip(qs, ks, mark[0]):
            k[key, :, mark[1]] *= 3.0
            q[-1, :, mark[1]] = k[key, :, mark[1]].repeat_interleave(heads // kvh, dim=0) * 1.5
    qs, ks, vs = ([t.to(rt.dtype).float() for t in x] for x in (qs, ks, vs))
    cache = torch.full((num_pages, 2, kvh, page, dp), float("nan"), dtype=rt.dtype, device=rt.device)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))  # noqa: E731
    K.fill_cache(cache, tables, [pad(k.reshape(k.shape[0], kvh, 2 * d), dp) for k in ks], [pad(v, dp) for v in vs], page)
    ctx, _ = K.make_context(rt, entries, page, tables)
    wide = torch.zeros(ctx.T, heads, 2, dp)
    q = torch.cat([x[c:c + n] for (c, n), x in zip(entries, qs)])
    wide[:, :, 0, :d], wide[:, :, 1, d:2 * d] = q[:, :, 0], q[:, :, 1]
    out = torch.full((ctx.T, heads * 2 * dp), float("nan"), dtype=rt.dtype, device=rt.device)
    rt.ops.scored_fast_attention = fast
    try:
        rt.ops.attention(wide.reshape(ctx.T, -1).to(rt.dtype).to(rt.device), heads * 2 * dp, cache, ctx, 0, out, 2 * heads, kvh, dp, page, num_pages,
                         window, 1 / math.sqrt(d), softcap=cap)
    finally:
        rt.ops.scored_fast_attention = True
    rt.ops.check_status()
    worst, row = 0.0, 0
    for (c, n), qq, k, v in zip(entries, qs, ks, vs):
        want = PX.two_maps(qq.double(), k.double(), v.double(), 1 / math.sqrt(d), cap or None, PX.visible(c + n, window or None))[c:]
        got = out[row:row + n].float().cpu().view(n, heads, 2, dp)
        worst = max(worst, float((got[..., :dv].double() - want).abs().max()))
        assert bool((got[..., dv:] == 0).all())
        row += n
    return worst


MAPS = [(4, 2, 24, 48, 16, 36, 4.0), (4, 1, 32, 64, 8, 64, 6.0), (6, 3, 8, 16, 4, 21, 0.0), (2, 1, 64, 128, 16, 100, 5.0), (4, 4, 20, 24, 8, 50, 3.0),
        (10, 1, 16, 32, 16, 40, 4.0), (2, 1, 64, 128, 16, 0, 8.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kvh,d,dv,page,window,cap", MAPS)
def test_two_maps_in_prompt_portions(rts, dtype, heads, kvh, d, dv, page, window, cap):
    """Portions that start and end anywhere, beside single tokens; for the last query of each request one key of one map
    towers: the newest outside its window, the oldest inside."""
    rt = rts[dtype]
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    W = window or 60
    entries = [(0, 3 * W + 5), (W - 2, 7), (2 * W - 1, 1), (W + 3, 2), (5, 2 * W), (0, 1), (1, 2)]
    for which in (0, 1):
        for m in (0, 1):
            keys = [min(max(c + n - 1 - W + which, 0), c + n - 1) for c, n in entries]
            for tc in (True, False) if dtype == "bfloat16" and max(2 * d, dv) in (64, 128) else (True,):
                rt.ops.tc_attention = tc
                try:
                    err = _maps_case(rt, entries, heads, kvh, d, dv, page, window, cap, seed=W + m, mark=(keys, m))
                finally:
                    rt.ops.tc_attention = True
                assert err < tol, (which, m, tc, err)


@pytest.mark.parametrize("dtype,fast", [("float32", True), ("bfloat16", True), ("bfloat16", False)])
@pytest.mark.parametrize("heads,kvh,d,dv,page,window,cap", MAPS)
def test_two_maps_in_decode_steps(rts, dtype, fast, heads, kvh, d, dv, page, window, cap):
    rt = rts[dtype]
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    W = window or 60
    entries = [(p, 1) for p in (0, 1, W - 1, W, W + 1, 3 * W + 7, 1500)]
    for which in (0, 1):
        for m in (0, 1):
            keys = [min(max(p - W + which, 0), p) for p, _ in entries]
            err = _maps_case(rt, entries, heads, kvh, d, dv, page, window, cap, seed=W + 2 + m, mark=(keys, m), fast=fast)
            assert err < tol, (which, m, err)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dv,dp", [(4, 48, 48), (3, 10, 32), (16, 128, 128), (2, 256, 256), (5, 30, 48), (1, 512, 512), (7, 100, 112), (2, 301, 304)])
def test_difference_norm_and_gate(rts, dtype, heads, dv, dp):
    """What lies behind a head's values in a padded result is never read (NaN there); without and with a gate."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(dv)
    T = 37
    ctx, _ = K.make_context(rt, [(0, 30), (3, 7)], 64, [[1], [2]])
    a = torch.randn(T, heads, 2, dp, generator=g).to(rt.dtype)
    a[3, :, 0, :dv] = (0.4 * a[3, :, 1, :dv].float()).to(rt.dtype)          # a near cancellation: eps decides
    gate = torch.randn(T, heads + 5, generator=g).to(rt.dtype)
    lam = torch.tensor([0.4])
    want = PX.difference(a[..., :dv].double(), lam.double(), 0.35, 1e-3)
    a[..., dv:] = float("nan")
    dev = lambda t: t.to(rt.device)  # noqa: E731
    for gv, ref in ((None, want), (gate, want * torch.sigmoid(gate[:, 5:].double())[:, :, None])):
        out = torch.full((T, heads * dv), float("nan"), dtype=rt.dtype, device=rt.device)
        rt.ops.map_difference(dev(a).view(T, -1), dev(gv)[:, 5:] if gv is not None else None, dev(lam), 0.65, 1e-3, out, ctx.meta, heads=heads, dp=dp)
        got = out.float().cpu().double().view(T, heads, dv)
        assert torch.allclose(got, ref, atol=(2e-5 if dtype == "float32" else 1e-2) * float(ref.abs().max()))
    rt.ops.check_status()
