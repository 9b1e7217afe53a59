"""The kernels that the Kavotar layers add or extend, alone against the plain functions: attention whose softmax weights are
mixed across heads (plain, decode and prefill kernels, one key made to tower just inside or just outside a chunk's edge),
attention rows with a scale per query head, the norm of a sublayer's result with its sum into the stream, the layer norm of
chosen rows, rows moved toward the token before, the scan with a bonus, the memory with exponential gates, the norm per head
with a weight per channel, and the router with sigmoid scores, a correction and groups."""
import math

import pytest
import torch

import kernel_utils as K
import plain_kavotar as PV
from atoma_infer_b200.parts.base import PendingSum

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


def _context(rt, cur, slots):
    ctx, _ = K.make_context(rt, [(a, c) for _, a, c in cur], 16, [[1]] * len(cur))
    ctx.state_slots.copy_(torch.tensor([slots[k] for k, _, _ in cur], dtype=torch.int32))
    return ctx


# ---------------------------------------------------------------------------------------------- weights mixed across heads
def _talk_case(rt, H, G, d, dv, page, chunk, lens, seed, tower=None):
    """Requests of the given lengths in a scrambled cache; returns what the kernels read and the plain outputs."""
    g = torch.Generator().manual_seed(seed)
    dp = -(-max(d, dv) // 16) * 16 if rt.dtype == torch.bfloat16 else max(d, dv)
    r = lambda *s: torch.randn(*s, generator=g).to(rt.dtype).double()  # noqa: E731  (values that the storage holds exactly)
    qs, ks, vs = [r(n, H, d) for n in lens], [r(n, G, d) for n in lens], [r(n, G, dv) for n in lens]
    if tower is not None:  # key ``tower`` of the first request answers every head's query far louder than any other
        ks[0][tower] = 2.0
        qs[0][:] = (qs[0].abs() * 0.25 + 0.5).to(rt.dtype).double()
        vs[0][tower] = 8.0
    talk = (torch.randn(H, H, generator=g) * 0.7).to(torch.bfloat16).double()
    scale = d ** -0.5 * 1.3
    want = []
    for q, k, v in zip(qs, ks, vs):
        p = PV.head_weights(q, k, scale, torch.ones(H, dtype=torch.float64), PV.visible(q.shape[0], chunk))
        want.append(PV.weighted_values(PV.mix_heads(p, talk), v))
    tables, num_pages = K.scrambled_tables(lens, page, seed=seed)
    pad = lambda x: torch.nn.functional.pad(x, (0, dp - x.shape[-1]))  # noqa: E731
    cache = torch.full((num_pages, 2, G, page, dp), float("nan"), dtype=rt.dtype, device=rt.device)
    K.fill_cache(cache, tables, [pad(k).to(rt.device) for k in ks], [pad(v).to(rt.device) for v in vs], page)
    return dp, [pad(q) for q in qs], cache, tables, num_pages, talk.float().to(rt.device), scale, want


def _talk_run(rt, entries, qs, dp, H, G, cache, tables, num_pages, page, chunk, scale, talk, **over):
    """``entries``: (request, context, tokens); returns the outputs per entry [tokens, H, dp]."""
    ctx, _ = K.make_context(rt, [(a, n) for _, a, n in entries], page, [tables[k] for k, _, _ in entries])
    for k, v in over.items():
        setattr(ctx, k, v)
    q = torch.cat([qs[k][a:a + n] for k, a, n in entries]).to(rt.dtype).to(rt.device).view(ctx.T, H * dp).contiguous()
    out = torch.full((ctx.T, H * dp), float("nan"), dtype=rt.dtype, device=rt.device)
    rt.ops.talking_attention(q, H * dp, cache, ctx, 0, out, H, G, dp, page, num_pages, scale, talk, chunk=chunk or 0)
    rt.ops.check_status()
    res, at = [], 0
    for _, _, n in entries:
        res.append(out[at:at + n].float().cpu().double().view(n, H, dp))
        at += n
    return res


TALK = [  # heads, key/value heads, key size, value size, page, chunk
    (4, 2, 16, 16, 4, 12), (8, 1, 64, 64, 16, None), (6, 3, 48, 32, 8, 25), (5, 5, 32, 16, 16, 64), (32, 8, 64, 64, 16, 96),
    (16, 16, 64, 64, 32, 50), (20, 1, 16, 32, 8, 40), (32, 4, 128, 128, 16, 70), (3, 1, 96, 80, 4, 33), (12, 4, 256, 200, 16, 30),
    (40, 8, 64, 64, 16, None), (1, 1, 32, 32, 16, 20),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,page,chunk", TALK)
def test_weights_mixed_across_heads(rts, dtype, H, G, d, dv, page, chunk):
    """Whole prompts, portions inside a cached context and decode steps of unequal requests, on the tensor-core kernels and
    on the plain one."""
    rt = rts[dtype]
    lens = (1, 17, 75, 140)
    dp, qs, cache, tables, num_pages, talk, scale, want = _talk_case(rt, H, G, d, dv, page, chunk, lens, seed=H + d)
    args = (qs, dp, H, G, cache, tables, num_pages, page, chunk, scale, talk)
    tol = 2e-6 * H if dtype == "float32" else 0.02
    big = max(float(w.abs().max()) for w in want)
    steps = [[(k, 0, n) for k, n in enumerate(lens)],                                        # whole prompts
             [(1, 3, 14), (2, 37, 2), (3, 60, 80), (0, 0, 1)],                               # portions cut anywhere
             [(k, n - 1, 1) for k, n in enumerate(lens)],                                    # a decode step
             [(3, 139, 1)], [(2, 49, 1), (3, 100, 1)]]
    for fast in ((True, False) if dtype == "bfloat16" else (True,)):
        rt.ops.fast_talking_attention = fast
        try:
            for entries in steps:
                for (k, a, n), got in zip(entries, _talk_run(rt, entries, *args)):
                    err = float((got[..., :dv] - want[k][a:a + n]).abs().max()) / big
                    assert err <= tol, (fast, entries, k, err)
                    assert not got[..., dv:].abs().max() > 0 if dp > dv else True
        finally:
            rt.ops.fast_talking_attention = True


@pytest.mark.parametrize("dtype,first", [("float32", 64), ("bfloat16", 1 << 30), ("bfloat16", 1)])
@pytest.mark.parametrize("chunk,page", [(24, 16), (32, 16), (7, 4), (50, 8)])
def test_a_towering_key_shows_inside_its_chunk_and_nowhere_else(rts, monkeypatch, dtype, first, chunk, page):
    """The key at a chunk's first place dominates every query of the chunk, to its last place, and none of the next chunk; in
    prompts, in portions that start inside the chunk, and in decode steps."""
    rt, H, G, d = rts[dtype], 8, 2, 64
    monkeypatch.setattr(rt.ops, "TALK_TC_FROM", first)
    tower = 2 * chunk
    n = 4 * chunk + 3
    dp, qs, cache, tables, num_pages, talk, scale, want = _talk_case(rt, H, G, d, d, page, chunk, (n,), seed=5, tower=tower)
    args = (qs, dp, H, G, cache, tables, num_pages, page, chunk, scale, talk)
    big = float(want[0].abs().max())
    whole = _talk_run(rt, [(0, 0, n)], *args)[0]
    loud = whole[3 * chunk - 1].abs().max(), whole[3 * chunk].abs().max(), whole[tower - 1].abs().max()
    assert loud[0] > 2 * loud[1] and loud[0] > 2 * loud[2], loud
    tol = 2e-5 if dtype == "float32" else 0.02
    assert float((whole - want[0]).abs().max()) <= tol * big
    for a, c in ((3 * chunk - 1, 2), (tower - 1, 2), (tower + 1, chunk), (3 * chunk - 2, 3)):
        got = _talk_run(rt, [(0, a, c)], *args)[0]
        assert float((got - want[0][a:a + c]).abs().max()) <= tol * big, (a, c)
    for a in (tower - 1, tower, tower + 1, 3 * chunk - 1, 3 * chunk, n - 1):
        got = _talk_run(rt, [(0, a, 1)], *args)[0]
        assert float((got - want[0][a:a + 1]).abs().max()) <= tol * big, a


TALK_LARGE = [  # heads, key/value heads, key and value size, page, chunk: what the tcgen05 kernels take
    (32, 8, 64, 16, 96), (16, 8, 64, 64, None), (8, 1, 128, 16, 130), (32, 4, 128, 16, 64), (6, 3, 64, 8, 37), (12, 4, 128, 32, None),
    (2, 2, 64, 128, 200), (40, 8, 64, 16, 90),  # (the last has more heads than slots: the kernels pass it on)
]


@pytest.mark.parametrize("H,G,d,page,chunk", TALK_LARGE)
def test_weights_mixed_across_heads_in_long_prompts(rts, H, G, d, page, chunk):
    """The tcgen05 kernels, forced for any number of tokens: prompts that end inside a tile, portions that start inside a
    chunk, a page and a tile, steps of unequal requests; against the plain outputs and against the other prefill kernel."""
    rt = rts["bfloat16"]
    lens = (1, 9, 128, 333)
    dp, qs, cache, tables, num_pages, talk, scale, want = _talk_case(rt, H, G, d, d, page, chunk, lens, seed=H + d + 1)
    args = (qs, dp, H, G, cache, tables, num_pages, page, chunk, scale, talk)
    big = max(float(w.abs().max()) for w in want)
    steps = [[(k, 0, n) for k, n in enumerate(lens)], [(3, 0, 333)],
             [(1, 3, 2), (2, 37, 91), (3, 131, 130), (0, 0, 1)], [(3, 127, 2), (2, 120, 8)], [(3, 261, 72)]]
    before, results = rt.ops.TALK_TC_FROM, {}
    try:
        for first in (1, 1 << 30):
            rt.ops.TALK_TC_FROM = first
            results[first] = [_talk_run(rt, entries, *args) for entries in steps]
    finally:
        rt.ops.TALK_TC_FROM = before
    for first, runs in results.items():
        for entries, outs in zip(steps, runs):
            for (k, a, n), got in zip(entries, outs):
                assert float((got - want[k][a:a + n]).abs().max()) / big <= 0.02, (first, entries, k)


def test_decode_steps_with_a_bound_above_the_context(rts):
    """A captured graph sizes its blocks by a bound on the context, not by the context: empty blocks of a cluster, and
    padded rows beyond the batch."""
    rt, H, G, d, page = rts["bfloat16"], 8, 2, 64, 16
    for chunk in (None, 400):
        dp, qs, cache, tables, num_pages, talk, scale, want = _talk_case(rt, H, G, d, d, page, chunk, (5, 530, 64), seed=9)
        args = (qs, dp, H, G, cache, tables, num_pages, page, chunk, scale, talk)
        entries = [(0, 4, 1), (1, 529, 1), (2, 63, 1)]
        for bound in (530, 1024, 2048):
            for (k, a, n), got in zip(entries, _talk_run(rt, entries, *args, max_context=bound)):
                assert float((got - want[k][a:a + n]).abs().max()) <= 0.02 * float(want[k].abs().max()), (chunk, bound, k)


# ---------------------------------------------------------------------------------------------- rows and norms
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,dv,rot", [(32, 16, 16), (18, 10, 6), (64, 64, 64), (24, 32, 0)])
def test_attention_rows_with_a_scale_per_query_head(rts, dtype, d, dv, rot):
    rt, H, G, page, eps = rts[dtype], 6, 2, 8, 1e-5
    g = torch.Generator().manual_seed(d)
    n, start, dp = 21, 9, -(-max(d, dv) // 16) * 16
    rows = torch.randn(n, H * d + G * d + G * dv, generator=g).to(rt.dtype)
    qn, kn, temp = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.5 * torch.randn(H, generator=g)
    inv = torch.tensor([500.0 ** (-2.0 * i / rot) for i in range(rot // 2)]) if rot else None
    tables, num_pages = K.scrambled_tables((start + n,), page, seed=1)
    ctx, _ = K.make_context(rt, [(start, n)], page, tables)
    cache = torch.full((num_pages, 2, G, page, dp), 9.0, dtype=rt.dtype, device=rt.device)
    q_out = torch.full((n, H * dp), float("nan"), dtype=rt.dtype, device=rt.device)
    rt.ops.qkv_prepare(rows.to(rt.device), ctx, cache, 0, q_out, nq=H, nkv=G, d=d, dv=dv, dp=dp, page_size=page, num_pages=num_pages,
                       store_kv=True, q_norm=qn.to(rt.device), k_norm=kn.to(rt.device), eps=eps, inv_freq=inv.to(rt.device) if rot else None,
                       rot=rot, head_norm=True, q_head_scale=temp.to(rt.device))
    rt.ops.check_status()
    x = rows.double()
    lead = torch.zeros((start, H, d), dtype=torch.float64)
    q = PV.rms(x[:, :H * d].view(n, H, d), eps) * qn.double()
    k = PV.rms(x[:, H * d:(H + G) * d].view(n, G, d), eps) * kn.double()
    q = PV.rotate_halves(torch.cat([lead, q]), rot, 500.0)[start:] * temp.double()[:, None]
    k = PV.rotate_halves(torch.cat([lead[:, :G], k]), rot, 500.0)[start:]
    tol = 2e-5 if dtype == "float32" else 3e-2
    got = q_out.float().cpu().double().view(n, H, dp)
    assert torch.allclose(got[..., :d], q, atol=tol, rtol=tol) and (dp == d or got[..., d:].abs().max() == 0)
    for i in range(n):
        page_id, slot = tables[0][(start + i) // page], (start + i) % page
        assert torch.allclose(cache[page_id, 0, :, slot, :d].float().cpu().double(), k[i], atol=tol, rtol=tol)
        assert torch.allclose(cache[page_id, 1, :, slot, :dv].float().cpu().double(), x[i, (H + G) * d:].view(G, dv), atol=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [40, 70, 256, 2048, 4100, 5120, 16384])
@pytest.mark.parametrize("layer_norm", [True, False])
def test_norm_of_a_result_with_its_sum_into_the_stream(rts, dtype, H, layer_norm):
    """One to three terms with weights, some normed over the width first, an offset that only the layer norm takes off, a
    vector, with and without the next input."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(H)
    T = 9
    ctx = _context(rt, [(0, 0, T)], [0])
    dev = lambda t: t.to(rt.device)  # noqa: E731
    w = 1 + 0.3 * torch.randn(H, generator=g)
    for factors, normed, vector in (((1.0,), (False,), False), ((0.5, 0.5), (True, True), False), ((0.3, -1.5, 0.8), (True, False, True), True)):
        terms = [(torch.randn(T, H, generator=g) * (3.0 if nm else 1.0) + 0.7).to(rt.dtype) for nm in normed]
        nws = [1 + 0.4 * torch.randn(H, generator=g) for _ in normed]
        vec = torch.randn(H, generator=g) if vector else None
        resid = torch.randn(T, H, generator=g)
        y = sum(f * (PV.rms(t.double(), 1e-3) * nw.double() if nm else t.double()) for f, t, nw, nm in zip(factors, terms, nws, normed))
        y = 1.25 * y + (vec.double() if vector else 0)
        want = resid.double() + (PV.layer_norm(y, w, 1e-5) if layer_norm else PV.rms(y, 1e-5) * w.double())
        for with_out in (True, False):
            r = dev(resid.clone())
            out = torch.full((T, H), float("nan"), dtype=rt.dtype, device=rt.device) if with_out else None
            pend = PendingSum(tuple(dev(t) for t in terms), 1.25, vector=dev(vec) if vector else None, factors=factors,
                              norms=tuple((dev(nw), 1e-3) if nm else None for nw, nm in zip(nws, normed)))
            rt.ops.norm_add(r, pend, dev(w), 1e-5, ctx, layer_norm=layer_norm, out=out)
            assert torch.allclose(r.cpu().double(), want, atol=2e-5, rtol=2e-5), (factors, float((r.cpu().double() - want).abs().max()))
            if with_out:
                assert torch.equal(out, r.to(rt.dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [37, 512, 3000])
def test_layer_norm_of_chosen_rows(rts, dtype, H):
    rt = rts[dtype]
    g = torch.Generator().manual_seed(H)
    x, w = torch.randn(12, H, generator=g) * 4 + 30, 1 + 0.3 * torch.randn(H, generator=g)
    ctx, rows = K.make_context(rt, [(0, 12)], 16, [[1]], rows=[11, 0, 7])
    out = torch.empty((3, H), dtype=rt.dtype, device=rt.device)
    rt.ops.layer_norm(x.to(rt.device), w.to(rt.device), 1e-5, out, ctx.meta, 3, rows=rows)
    tol = 5e-5 if dtype == "float32" else 2e-2
    assert torch.allclose(out.float().cpu().double(), PV.layer_norm(x.double(), w, 1e-5)[[11, 0, 7]], atol=tol, rtol=tol)
    allrows = torch.empty((12, H), dtype=rt.dtype, device=rt.device)
    rt.ops.layer_norm(x.to(rt.device), w.to(rt.device), 1e-5, allrows, ctx.meta, 12)
    assert torch.allclose(allrows.float().cpu().double(), PV.layer_norm(x.double(), w, 1e-5), atol=tol, rtol=tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [38, 256, 1100])
def test_rows_moved_toward_the_token_before(rts, dtype, H):
    """Portions of 1, 2 and more tokens in one batch and steps of single tokens; the kept row lives in scattered slots that
    are slices of a wider state; a slot that held another request's row reads as zeros at position 0."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(H)
    lens = [23, 5, 31]
    xs, mu = [torch.randn(n, H, generator=g) for n in lens], torch.rand(3, H, generator=g) * 1.3
    want = [torch.stack([PV.moved_toward_previous(x.double(), m) for m in mu]) for x in xs]
    slots = [3, 0, 1]
    state = torch.full((4, 8 + H + 4), 7.0, device=rt.device)[:, 8:8 + H]
    tol = 1e-5 if dtype == "float32" else 2e-2
    saved = set()
    for cur in _portions(lens, (3, 1, 2, 7, 1, 1)):
        ctx = _context(rt, cur, slots)
        x = torch.cat([xs[k][a:a + c] for k, a, c in cur]).to(rt.device)
        out = torch.full((3, ctx.T, H), float("nan"), dtype=rt.dtype, device=rt.device)
        done = rt.ops.token_mix(x, mu.to(rt.device), state, ctx, out)
        saved.add(done)
        if not done:
            rt.ops.keep_last_rows(x, state, ctx)
        r = 0
        for k, a, c in cur:
            assert torch.allclose(out[:, r:r + c].float().cpu().double(), want[k][:, a:a + c], atol=tol, rtol=tol), (k, a, c)
            assert torch.equal(state[slots[k]].cpu(), xs[k][a + c - 1])
            r += c
    assert saved == {True, False}


# ---------------------------------------------------------------------------------------------- recurrences
SCAN = [(2, 16, 16), (3, 24, 40), (1, 72, 72), (5, 10, 14), (2, 64, 64), (1, 128, 256), (4, 8, 33), (2, 48, 48)]


def _scan_steps(lens, long_first):
    return _portions(lens, (150, 2, 200, 1, 64)) if long_first else _portions(lens, (3, 1, 2, 17, 1, 40))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", SCAN)
@pytest.mark.parametrize("chunked", [False, True])
def test_scan_with_a_bonus_over_portions_and_slots(rts, dtype, heads, dim, vdim, chunked):
    """Decays from none to all at once, one channel that forgets nothing and keeps an early, loud key; in order and in
    chunks of time."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(heads * dim)
    lens = [300, 190, 130] if chunked else [61, 5, 33]
    K_, V_ = heads * dim, heads * vdim
    r = lambda n, c, s=1.0: (torch.randn(n, c, generator=g) * s).to(rt.dtype)  # noqa: E731
    rs, ks, vs = [r(n, K_) for n in lens], [r(n, K_, 0.5) for n in lens], [r(n, V_) for n in lens]
    zs = [torch.randn(n, K_, generator=g) * 2.0 - 2.0 for n in lens]
    w0, u = torch.randn(K_, generator=g), torch.randn(K_, generator=g)
    for z in zs:
        z[:, 1] = -30.0 - w0[1]  # this channel of the first head forgets nothing
        z[:, 2] = 8.0 - w0[2]    # and this one everything
    ks[0][2, 1] = 4.0
    want = []
    for a, b, c, z in zip(rs, ks, vs, zs):
        n = a.shape[0]
        decay = torch.exp(-torch.exp(z.double() + w0.double())).view(n, heads, dim)
        args = a.double().view(n, heads, dim), b.double().view(n, heads, dim), c.double().view(n, heads, vdim)
        want.append(PV.bonus_state(*args, decay, u.double().view(heads, dim)).reshape(n, V_))
    slots, wide = [2, 0, 3], torch.full((4, 12 + heads * dim * vdim + 8), 5.0, device=rt.device)
    state = wide[:, 12:12 + heads * dim * vdim].view(4, heads, dim, vdim)
    state.zero_()
    tol = 3e-5  # (in both types: inputs are what the storage holds; everything after is float32)
    for cur in _scan_steps(lens, chunked):
        ctx = _context(rt, cur, slots)
        cat = lambda xs: torch.cat([xs[k][a:a + c] for k, a, c in cur]).to(rt.device)  # noqa: E731
        rows = torch.cat([cat(rs), cat(ks), cat(vs)], 1).contiguous()
        o = torch.full((ctx.T, V_), float("nan"), device=rt.device)
        rt.ops.bonus_scan(rows[:, :K_], rows[:, K_:2 * K_], rows[:, 2 * K_:], cat(zs), w0.to(rt.device), u.to(rt.device), state, ctx, o,
                          heads=heads, dim=dim, vdim=vdim)
        at = 0
        for k, a, c in cur:
            err = float((o[at:at + c].cpu().double() - want[k][a:a + c]).abs().max()) / float(want[k].abs().max())
            assert err <= tol, (k, a, c, err)
            at += c
    assert float(wide[:, :12].min()) == 5.0 and float(wide[:, -8:].max()) == 5.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", SCAN)
@pytest.mark.parametrize("chunked", [False, True])
def test_memory_with_exponential_gates_over_portions_and_slots(rts, dtype, heads, dim, vdim, chunked):
    """Gates that open and close by many orders of magnitude, a normalizer below and above its floor, an early token whose
    input gate towers and is remembered; the running maximum starts at 0 and crosses portions; in order and in chunks."""
    rt = rts[dtype]
    g = torch.Generator().manual_seed(heads * dim + 1)
    lens = [300, 190, 290] if chunked else [61, 5, 33]
    K_, V_, cap = heads * dim, heads * vdim, 7.0
    r = lambda n, c, s=1.0: (torch.randn(n, c, generator=g) * s).to(rt.dtype)  # noqa: E731
    qs, ks, vs, gs = [r(n, K_) for n in lens], [r(n, K_) for n in lens], [r(n, V_) for n in lens], [r(n, V_) for n in lens]
    xs = [torch.randn(n, 2 * heads, generator=g) * 4.0 for n in lens]
    bias = torch.cat([torch.randn(heads, generator=g), 3 + torch.randn(heads, generator=g)])
    xs[0][3, 0] = 40.0             # a towering input gate (capped), kept by forget gates near 1 ...
    xs[0][4:40, heads] = 30.0
    xs[2][0, 0] = -40.0            # ... and a first token that hardly enters: m stays at 0, the floor is 1
    w = 1 + 0.3 * torch.randn(V_, generator=g)
    want, want_n = [], []
    for a, b, c, x, gate in zip(qs, ks, vs, xs, gs):
        n = a.shape[0]
        z = PV.soft_limit(x.double() + bias.double(), cap)
        o = PV.matrix_memory(a.double().view(n, heads, dim) * dim ** -0.5, b.double().view(n, heads, dim), c.double().view(n, heads, vdim),
                             z[:, :heads], PV.log_sigmoid(z[:, heads:]))
        want.append(o.reshape(n, V_))
        want_n.append(PV.rms(o, 1e-5).reshape(n, V_) * w.double() * torch.sigmoid(gate.double()))
    slots, S = [2, 0, 3], heads * dim * vdim
    up = lambda n: -(-n // 4) * 4  # noqa: E731
    wide = torch.full((4, 12 + up(S) + up(K_) + up(heads) + 8), 5.0, device=rt.device)
    state, n_state = wide[:, 12:12 + S].view(4, heads, dim, vdim), wide[:, 12 + up(S):12 + up(S) + K_].view(4, heads, dim)
    m_state = wide[:, 12 + up(S) + up(K_):12 + up(S) + up(K_) + heads]
    for t in (state, n_state, m_state):
        t.zero_()
    for cur in _scan_steps(lens, chunked):
        ctx = _context(rt, cur, slots)
        cat = lambda ys: torch.cat([ys[k][a:a + c] for k, a, c in cur]).to(rt.device)  # noqa: E731
        rows = torch.cat([cat(qs), cat(ks), cat(vs), cat(gs)], 1).contiguous()
        o = torch.full((ctx.T, V_), float("nan"), device=rt.device)
        nq, floor = torch.full((ctx.T, heads), float("nan"), device=rt.device), torch.full((ctx.T, heads), float("nan"), device=rt.device)
        rt.ops.memory_scan(rows[:, :K_], rows[:, K_:2 * K_], rows[:, 2 * K_:2 * K_ + V_], cat(xs).contiguous(), bias.to(rt.device), cap,
                           dim ** -0.5, state, n_state, m_state, ctx, o, nq, floor, heads=heads, dim=dim, vdim=vdim)
        y = torch.full((ctx.T, V_), float("nan"), dtype=rt.dtype, device=rt.device)
        rt.ops.head_weight_norm_gate(o, rows[:, 2 * K_ + V_:], w.to(rt.device), 1e-5, y, ctx.meta, heads, kind="sigmoid", nq=nq, floor=floor)
        den = torch.maximum(nq.abs(), floor) + 1e-6
        got = (o.view(ctx.T, heads, vdim) / den[:, :, None]).reshape(ctx.T, V_).cpu().double()
        at = 0
        for k, a, c in cur:
            # (a quotient of two sums: judged where the normalizer does not cancel, by the head's own size there)
            err = (got[at:at + c] - want[k][a:a + c]).abs() / (want[k][a:a + c].abs().amax(-1, keepdim=True) + 0.05)
            assert float(err.max()) <= 2e-3 and float(err.median()) <= 1e-5, (k, a, c, float(err.max()))
            n_err = (y[at:at + c].float().cpu().double() - want_n[k][a:a + c]).abs().max()
            assert float(n_err) <= (1e-3 if dtype == "float32" else 6e-2), (k, a, c, float(n_err))
            at += c


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,P", [(1, 24), (3, 10), (5, 64), (16, 128), (2, 33)])
@pytest.mark.parametrize("kind", ["sigmoid", "silu"])
def test_norm_per_head_with_a_weight_per_channel(rts, dtype, heads, P, kind):
    rt = rts[dtype]
    g = torch.Generator().manual_seed(heads * P)
    T, n = 7, heads * P
    o, w = torch.randn(T, n, generator=g) * 2, 1 + 0.4 * torch.randn(n, generator=g)
    wide = torch.randn(T, n + 24, generator=g).to(rt.dtype)
    ctx = _context(rt, [(0, 0, T)], [0])
    out = torch.empty((T, n), dtype=rt.dtype, device=rt.device)
    rt.ops.head_weight_norm_gate(o.to(rt.device), wide.to(rt.device)[:, 8:8 + n], w.to(rt.device), 1e-3, out, ctx.meta, heads, kind=kind)
    gate = wide[:, 8:8 + n].double()
    want = PV.rms(o.double().view(T, heads, P), 1e-3).reshape(T, n) * w.double() * (PV.silu(gate) if kind == "silu" else torch.sigmoid(gate))
    tol = 1e-5 if dtype == "float32" else 2e-2
    assert torch.allclose(out.float().cpu().double(), want, atol=tol, rtol=tol)


# ---------------------------------------------------------------------------------------------- router
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,groups", [(16, 3, (4, 3)), (8, 2, None), (12, 5, (4, 2)), (9, 4, (3, 3)), (6, 2, (6, 3)), (64, 8, (8, 4)),
                                                (256, 8, (8, 4)), (5, 5, None), (96, 6, (48, 5)), (3, 1, (1, 1))])
def test_router_with_sigmoid_scores_a_correction_and_groups(rts, dtype, experts, top, groups):
    """Corrections large enough to make choice scores negative and to turn choices; weights without them."""
    rt, H, T = rts[dtype], 136, 50
    g = torch.Generator().manual_seed(experts)
    h, w = torch.randn(T, H, generator=g).to(rt.dtype), torch.randn(experts, H, generator=g) * 0.15
    corr = torch.randn(experts, generator=g) * 0.8 - 0.5
    ctx = _context(rt, [(0, 0, T)], [0])
    ids = torch.full((T, top), -1, dtype=torch.int32, device=rt.device)
    wts = torch.full((T, top), float("nan"), device=rt.device)
    rt.ops.moe_route_sigmoid(h.to(rt.device), w.to(rt.device), corr.to(rt.device), ids, wts, ctx.meta, groups=groups)
    margins: list = []
    s = torch.sigmoid(h.double() @ w.double().T)
    idx, wt = PV.choose(s, corr, top, {"count": groups[0], "keep": groups[1]} if groups else None, margins)
    clear = margins[0] > 1e-5
    assert clear.sum() > T * 0.8
    assert torch.equal(ids.cpu().long().sort(1).values[clear], idx.sort(1).values[clear])
    got = torch.gather(s, 1, ids.cpu().long())
    assert torch.allclose(wts.cpu().double(), got, atol=1e-6)  # (every weight is its own expert's score)


def test_router_ties_go_to_the_lower_index(rts):
    rt, H, E = rts["float32"], 32, 8
    h, w = torch.zeros(2, H), torch.zeros(E, H)
    corr = torch.tensor([0.0, 0.5, 0.5, 0.0, 0.5, 0.5, 0.0, 0.0])
    ctx = _context(rt, [(0, 0, 2)], [0])
    ids, wts = torch.zeros((2, 3), dtype=torch.int32, device=rt.device), torch.zeros((2, 3), device=rt.device)
    rt.ops.moe_route_sigmoid(h.to(rt.device), w.to(rt.device), corr.to(rt.device), ids, wts, ctx.meta, groups=(4, 2))
    # groups {0,1} {2,3} {4,5} {6,7}: sums 1.5, 1.5, 2.0, 1.0 -> {4,5} and, of the two that tie, {0,1}
    assert ids.cpu().tolist() == [[1, 4, 5]] * 2 and torch.allclose(wts.cpu(), torch.full((2, 3), 0.5))
