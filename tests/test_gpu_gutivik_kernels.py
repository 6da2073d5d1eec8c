"""The kernels of attention over convolved projections, gated linear attention and router-chosen experts, each against the plain
restatement of its mechanism."""
import math

import pytest
import torch

from oracles import gutivik as O

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
DTYPES = [(F32, 3e-6), (BF, 6e-3)]


def _m():
    from nexus_b200.ops import _mixers as M
    return M


def _x():
    from nexus_b200.ops import _experts as X
    return X


def _rand(shape, seed, dtype=F32, s=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s).to(dtype)


def _err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).norm() / want.norm().clamp_min(1e-30)).item()


def _segs(parts):
    """parts: (first row, rows, first position, slot) per segment."""
    t = torch.tensor(parts, dtype=torch.int32).t().contiguous()
    return _m().Segments(t.to(DEV), 0, len(parts), max(p[1] for p in parts), sum(p[1] for p in parts))


def _tables(rot, n):
    ang = torch.arange(n).double()[:, None] * torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)],
                                                           dtype=torch.float64)
    return ang.cos().float().to(DEV), ang.sin().float().to(DEV)


# ---------------------------------------------------------------------------------------------- residual stream, latents
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("cols", [96, 50, 2048])
def test_outputs_added_without_a_norm(dt, tol, cols):
    M = _m()
    n, top, slots, ld, eps = 7, 3, 30, (cols + 7) // 8 * 8, 1e-3
    x, y, rows = _rand((n, cols), 1), _rand((n, ld), 2, dt), _rand((slots, ld), 3, dt)
    wn, weights = 1 + _rand((cols,), 4, s=0.3), torch.rand((n, top), generator=torch.Generator().manual_seed(5))
    pick = torch.randint(0, slots, (n, top), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    want = x.double() + y[:, :cols].double()
    xd, h = x.clone().to(DEV), torch.full((n, ld), 7.0, dtype=dt, device=DEV)
    M.residual_norm(xd, y=y.to(DEV), w_next=wn.to(DEV), h=h, eps=eps)
    assert _err(xd, want) < 1e-6 and _err(h[:, :cols], O.rms(want, eps) * wn.double()) < tol and h[:, cols:].abs().sum() == 0
    want = want + (rows[pick.long()].double()[:, :, :cols] * weights.double()[:, :, None]).sum(1)
    M.residual_norm(xd, experts=rows.to(DEV), slots=pick.to(DEV), top=top, weights=weights.to(DEV), w_next=wn.to(DEV), h=h, eps=eps)
    assert _err(xd, want) < 1e-6 and _err(h[:, :cols], O.rms(want, eps) * wn.double()) < tol
    M.residual_norm(xd, y=y.to(DEV), res_mult=0.5, eps=eps)
    assert _err(xd, want + 0.5 * y[:, :cols].double()) < 1e-6


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_latent_prep_without_query_latent_and_gate(dt, tol):
    M = _m()
    n, rank, dims, row, eps = 9, 37, 6, 64, 1e-3
    proj, w = _rand((n, 88), 1, dt), 1 + _rand((rank,), 2, s=0.3)
    cos, sin = _tables({"dims": dims, "base": 50.0}, n)
    cache, lat = torch.zeros((4, 4, 1, row), dtype=dt, device=DEV), torch.full((n, row), 7.0, dtype=dt, device=DEV)
    M.latent_prep(proj.to(DEV), (0, 24, 64, 0), 0, rank, dims, 5, None, w.to(DEV), torch.arange(n, dtype=torch.int32, device=DEV),
                  torch.arange(n, dtype=torch.int32, device=DEV), cos, sin, None, cache, 48, None, eps=eps, lat=lat)
    c = O.rms(proj[:, 24: 24 + rank].double(), eps) * w.double()
    pairs = torch.stack([proj[:, 64: 67], proj[:, 67: 70]], -1).reshape(n, 1, dims).double()        # halves as neighbours
    r = O.rotate(pairs, {"dims": dims, "base": 50.0})[:, 0]
    want = torch.cat([c, torch.zeros(n, 48 - rank), r[:, 0::2], r[:, 1::2], torch.zeros(n, row - 48 - dims)], 1)
    assert _err(lat, want) < tol and _err(cache.view(-1, row)[:n], want) < tol


# ---------------------------------------------------------------------------------------------- convolution, rotation, mixing
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("taps,H,G,D,Dv,rot", [(1, 2, 1, 8, 4, 8), (2, 6, 3, 12, 20, 6), (3, 4, 4, 16, 8, 0), (4, 8, 2, 64, 32, 30), (7, 3, 1, 20, 24, 10)])
def test_conv_rope_append(dt, tol, taps, H, G, D, Dv, rot):
    """Two sequences in portions: what the whole sequence gives, in y and in the pages, first values written, then mixed."""
    M = _m()
    T, bs, C = 75, 4, H * D + G * (D + Dv)
    rotary = {"dims": rot, "base": 90.0}
    w, mix = _rand((C, taps), 2, s=0.6), 0.3
    cos, sin = _tables(rotary, T) if rot else (torch.zeros((T, 1), device=DEV),) * 2
    ld = -(-C // 8) * 8 + 8
    for cuts in ([T], [2, 3, 33, 1, 1, 35], [1] * 9 + [T - 9]):
        tail = torch.full((3, max(taps - 1, 1), C), 9.0, dtype=dt, device=DEV)
        kc, vc = torch.zeros((40, bs, G, D), dtype=dt, device=DEV), torch.zeros((40, bs, G, Dv), dtype=dt, device=DEV)
        xs = [_rand((T, C), 10 + len(cuts) + i, dt) for i in range(2)]
        first = [_rand((T, G * Dv), 30 + i, dt) for i in range(2)]
        want = []
        for i in range(2):
            u = O.causal_conv(xs[i].double(), w.double())
            q, k, v = u.split([H * D, G * D, G * Dv], 1)
            q, k = (O.rotate(t.reshape(T, -1, D), rotary).reshape(T, -1) if rot else t for t in (q, k))
            want.append((q, k, v, v if i == 0 else (1 - mix) * v + mix * first[i].double()))
        place = [list(range(5, 5 + T)), list(range(80, 80 + T))]       # cache slot of every position
        got, pos = [[], []], 0
        for n in cuts:
            x = torch.zeros((2 * n + 1, ld), dtype=dt)
            x[:n, :C], x[n + 1:, :C] = xs[0][pos: pos + n], xs[1][pos: pos + n]
            slots = torch.tensor(place[0][pos: pos + n] + [-1] + place[1][pos: pos + n], dtype=torch.int32, device=DEV)
            y, x = torch.zeros((2 * n + 1, C), dtype=dt, device=DEV), x.to(DEV)[:, :C]
            f = torch.cat([torch.zeros(n + 1, G * Dv, dtype=dt), first[1][pos: pos + n]]).to(DEV)
            kw = dict(heads=H, kv_heads=G, dim=D, vdim=Dv, rot_dims=rot, cos_t=cos, sin_t=sin, slots=slots, k_cache=kc, v_cache=vc)
            wd = w.t().contiguous().to(DEV)
            M.conv_rope_append(x, y, wd, None, tail, _segs([(0, n, pos, 2)]), store_kv=True, first=f, **kw)
            M.conv_rope_append(x, y, wd, None, tail, _segs([(n + 1, n, pos, 0)]), first=f, mix=torch.tensor([mix], device=DEV), **kw)
            assert _err(f[:n], want[0][2][pos: pos + n]) < tol
            got[0].append(y[:n])
            got[1].append(y[n + 1:])
            assert y[n].abs().sum() == 0
            pos += n
        q0 = torch.cat(got[0])
        assert _err(q0, torch.cat([want[0][0], want[0][1], want[0][3]], 1)) < tol
        q1 = torch.cat(got[1])
        assert _err(q1[:, : H * D], want[1][0]) < tol and q1[:, H * D:].abs().sum() == 0
        for i in range(2):
            at = torch.tensor(place[i], device=DEV)
            assert _err(kc.view(-1, G * D)[at], want[i][1]) < tol and _err(vc.view(-1, G * Dv)[at], want[i][3]) < tol
        assert kc.view(-1, G * D)[:5].abs().sum() == 0


# ---------------------------------------------------------------------------------------------- attention
def _paged(lengths, bs, G, D, Dv, dt, seed=0):
    """Shuffled pages: caches, block table, and the keys and values of every sequence."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // bs) for n in lengths]
    pages = torch.randperm(sum(per) + 3, generator=g)
    kc, vc = torch.full((len(pages), bs, G, D), 90.0, dtype=dt), torch.full((len(pages), bs, G, Dv), 90.0, dtype=dt)
    table, ks, vs, p = torch.zeros((len(lengths), max(per) + 1), dtype=torch.int32), [], [], 0
    for i, n in enumerate(lengths):
        k, v = torch.randn(n, G, D, generator=g).to(dt), torch.randn(n, G, Dv, generator=g).to(dt)
        ks.append(k)
        vs.append(v)
        for b in range(per[i]):
            table[i, b] = pages[p]
            part = slice(b * bs, min(n, (b + 1) * bs))
            kc[pages[p], : part.stop - part.start], vc[pages[p], : part.stop - part.start] = k[part], v[part]
            p += 1
    return kc, vc, table, ks, vs


def _reference(q, ks, vs, segs, H, scale, window, keep, sink):
    out = torch.zeros((q.shape[0], H, vs[0].shape[2]), dtype=torch.float64)
    for r0, n, p0, seq in segs:
        k, v = ks[seq][: p0 + n].double(), vs[seq][: p0 + n].double()
        full = torch.zeros((p0 + n, H, k.shape[2]), dtype=torch.float64)
        full[p0:] = q[r0: r0 + n].double().view(n, H, -1)
        out[r0: r0 + n] = O.window_attention(full, k, v, scale, window if window else 1 << 30, keep, sink.double())[p0:]
    return out.view(q.shape[0], -1)


@pytest.mark.parametrize("window,keep", [(0, 0), (1, 1), (33, 6), (70, 64), (64, 65), (40, 130), (130, 3), (500, 9)])
@pytest.mark.parametrize("H,G,D,Dv,bs", [(6, 2, 24, 40, 16), (4, 4, 64, 64, 4), (20, 1, 128, 16, 24), (3, 3, 200, 8, 16)])
def test_paged_window_attention_with_kept_keys_and_sinks(H, G, D, Dv, bs, window, keep):
    """Decoding and portions in BF16, with and without spans of the keys, and FP32."""
    M = _m()
    lengths, scale, sink = [150, 1, 64, 65], 0.9 * D ** -0.5, _rand((H,), 9, s=2.0)
    for dt in (BF, F32):
        kc, vc, table, ks, vs = _paged(lengths, bs, G, D, Dv, dt)
        for segs, splits in (([(0, 1, 149, 0), (2, 1, 0, 1), (1, 1, 63, 2), (3, 1, 64, 3)], (1, 3)),
                             ([(0, 13, 137, 0), (14, 2, 0, 2), (16, 60, 5, 3)], (1,))):
            n = max(s[0] + s[1] for s in segs)
            q = _rand((n, H * D), 7, dt)
            want = _reference(q, ks, vs, segs, H, scale, window, keep, sink)
            live = torch.tensor(sorted(r for s in segs for r in range(s[0], s[0] + s[1])))
            for sp in splits:
                out = torch.full((n, H * Dv), 7.0, dtype=dt, device=DEV)
                M.paged_window_attention(q.to(DEV), kc.to(DEV), vc.to(DEV), table.to(DEV), out, _segs(segs), heads=H, block_size=bs,
                                         window=window, scale=scale, splits=sp, keep_first=keep, sink=sink.to(DEV))
                assert _err(out[live.to(DEV)], want[live]) < (6e-3 if dt == BF else 5e-6), (segs, sp, dt)


def _probe(window, keep, key, T):
    """Positions at which a key comes into, stays in, or has left the view of a query."""
    return [p for p in sorted({key, key + 1, key + window - 1, key + window, key + window + 1, T - 1}) if key <= p < T]


@pytest.mark.parametrize("window,keep", [(17, 5), (64, 16), (100, 33), (16, 0)])
def test_one_key_stands_out(window, keep):
    """A key that answers far above all others: its value is the output while it is in the window or among the kept first ones,
    and not one token later; with portions, decoding and the tcgen05 prompt kernel."""
    M = _m()
    H, G, D, Dv, bs, T = 2, 1, 64, 64, 16, 330
    kc, vc, table, ks, vs = _paged([T], bs, G, D, Dv, BF)
    sink = torch.zeros(H, device=DEV)
    for key in sorted({0, keep - 1, keep, 15, 16, 31, 99, 150, 255} - {-1}):
        poss = _probe(window, keep, key, T)
        q = torch.stack([ks[0][key, 0].float() * 4 for _ in poss]).to(BF).repeat(1, H).to(DEV)
        see = [p - key < window or key < keep for p in poss]

        def check(out):
            for i in range(len(poss)):
                hit = _err(out[i].view(H, Dv), vs[0][key].expand(H, -1)) < 2e-2
                assert hit == see[i], (key, poss[i])
        kw = dict(heads=H, window=window, scale=1.0, keep_first=keep, sink=sink)
        for splits in (1, 3):
            out = torch.zeros((len(poss), H * Dv), dtype=BF, device=DEV)
            M.paged_window_attention(q, kc.to(DEV), vc.to(DEV), table.to(DEV), out, _segs([(i, 1, p, 0) for i, p in enumerate(poss)]),
                                     block_size=bs, splits=splits, **kw)
            check(out)
        # as rows of a prompt and of a portion that starts in its middle
        for start in (0, 23, 140, 200):
            rows = [(i, p - start) for i, p in enumerate(poss) if p >= start]
            if not rows:
                continue
            full = _rand((T - start, H * D), 3, BF).to(DEV)
            for i, r in rows:
                full[r] = q[i]
            out = torch.zeros((T - start, H * Dv), dtype=BF, device=DEV)
            M.paged_window_attention(full, kc.to(DEV), vc.to(DEV), table.to(DEV), out, _segs([(0, T - start, start, 0)]), block_size=bs, **kw)
            other = torch.zeros_like(out)
            _prompt(full, kc, vc, table, [(0, T - start, start, 0)], other, dim=D, vdim=Dv, kv_heads=G, **kw)
            for o in (out, other):
                for i, r in rows:
                    hit = _err(o[r].view(H, Dv), vs[0][key].expand(H, -1)) < 2e-2
                    assert hit == see[i], (key, poss[i], start)


def _prompt(q, kc, vc, table, segs, out, *, window, keep_first, kv_heads, dim, vdim, fresh=None, **kw):
    """The prompt kernel over gathered keys, as the engine calls it (``fresh``: the rows of the step instead)."""
    from nexus_b200.infer.prompt import long_segments
    M = _m()
    blocks, runs, rows = long_segments(segs, window, keep_first if window else 0)
    if rows:
        k, v = torch.empty((rows, kv_heads * dim), dtype=BF, device=DEV), torch.empty((rows, kv_heads * vdim), dtype=BF, device=DEV)
        r = torch.tensor(runs, dtype=torch.int32, device=DEV)
        for c, dst in ((kc, k), (vc, v)):
            M.latent_gather(c.to(DEV), table.to(DEV), r, max(x[1] for x in runs), dst)
    else:
        if fresh is None:
            k, v = _rows_of(kc, table, segs, q.shape[0]), _rows_of(vc, table, segs, q.shape[0])
        else:
            k, v = fresh
    t = torch.tensor(blocks, dtype=torch.int32)
    M.window_prompt(q, k, v, out, t[:, :4].contiguous().to(DEV), kv_heads=kv_heads, dim=dim, vdim=vdim, window=window,
                    keep_first=keep_first, kept=t[:, 4].contiguous().to(DEV), **kw)


def _rows_of(cache, table, segs, n):
    """Keys or values of fresh segments in the row order of the step."""
    flat = cache.view(-1, cache.shape[2] * cache.shape[3])
    out = torch.zeros((n, flat.shape[1]), dtype=cache.dtype)
    bs = cache.shape[1]
    for r0, count, _, seq in segs:
        for j in range(count):
            out[r0 + j] = flat[int(table[seq, j // bs]) * bs + j % bs]
    return out.to(DEV)


@pytest.mark.parametrize("window,keep", [(0, 0), (1, 1), (40, 6), (129, 128), (64, 130), (300, 5), (20, 400)])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 64, 64), (6, 1, 128, 128), (3, 3, 16, 8), (8, 2, 96, 40), (2, 2, 48, 128)])
def test_window_prompt(H, G, D, Dv, window, keep):
    """Segments of many lengths packed beside one another: fresh ones, and portions behind earlier tokens."""
    M = _m()
    lengths, bs, sink, scale = [320, 700, 17, 300], 16, _rand((H,), 9, s=2.0), D ** -0.5
    kc, vc, table, ks, vs = _paged(lengths, bs, G, D, Dv, BF)
    for segs in ([(0, 320, 0, 0), (320, 700, 0, 1), (1022, 17, 0, 2)], [(3, 129, 191, 0), (132, 513, 187, 1), (645, 300, 0, 3)]):
        n = max(s[0] + s[1] for s in segs)
        q = _rand((n, H * D), 7, BF)
        want = _reference(q, ks, vs, segs, H, scale, window, keep, sink)
        live = torch.tensor(sorted(r for s in segs for r in range(s[0], s[0] + s[1])))
        out = torch.full((n, H * Dv), 7.0, dtype=BF, device=DEV)
        _prompt(q.to(DEV), kc, vc, table, segs, out, window=window, keep_first=keep, kv_heads=G, dim=D, vdim=Dv, heads=H, scale=scale,
                sink=sink.to(DEV))
        assert _err(out[live.to(DEV)], want[live]) < 6e-3, segs
        rest = torch.ones(n, dtype=torch.bool)
        rest[live] = False
        assert (out[rest.to(DEV)] == 7.0).all()
    from nexus_b200.ops import _cuda as K
    K.check_status()


# ---------------------------------------------------------------------------------------------- recurrence
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("rank,cols,tau", [(1, 7, 1.0), (5, 130, 16.0), (40, 256, 0.5)])
def test_decay_gate(dt, tol, rank, cols, tau):
    M = _m()
    a, w, b = _rand((70, rank + 3), 1, dt), _rand((cols, rank), 2), _rand((cols,), 3, s=20.0)
    got = M.decay_gate(a.to(DEV)[:, :rank], w.to(DEV), b.to(DEV), tau)
    want = O.log_sigmoid(a[:, :rank].double() @ w.double().t() + b.double()) / tau / math.log(2)
    assert _err(got, want) < 2e-6 and (got <= 0).all()
    far = want > -1e-6                       # decays next to one keep their distance from it
    assert _err(got.cpu()[far], want[far]) < 1e-4


def _gla_inputs(T, H, D, Dv, dt, seed, strength):
    q, k, v = _rand((T, H * D), seed, dt), _rand((T, H * D), seed + 1, dt), _rand((T, H * Dv), seed + 2, dt)
    z = _rand((T, H * D), seed + 3, s=2.0) + torch.linspace(-3.0, 4.0, D).repeat(H)
    dec = (O.log_sigmoid(z.double()) * strength).float()
    o = O.decayed_outer(q.double().view(T, H, D) * D ** -0.5, k.double().view(T, H, D), v.double().view(T, H, Dv), dec.double().view(T, H, D))
    S = torch.zeros(H, D, Dv, dtype=torch.float64)
    for t in range(T):
        S = torch.exp(dec[t].double()).view(H, D, 1) * S + k[t].double().view(H, D, 1) * v[t].double().view(H, 1, Dv)
    return q, k, v, dec / math.log(2), o.reshape(T, H * Dv), S


@pytest.mark.parametrize("strength", [0.06, 1.0, 9.0])
@pytest.mark.parametrize("H,D,Dv", [(3, 24, 20), (2, 64, 128), (4, 10, 7), (1, 72, 200), (2, 200, 64)])
@pytest.mark.parametrize("dt,tol,chunked", [(F32, 3e-6, False), (BF, 6e-3, False), (BF, 6e-3, True)])
def test_gla(H, D, Dv, dt, tol, chunked, strength):
    """Cut anywhere, in spans, from weak decays to ones that forget within a token; slots that held other states."""
    M = _m()
    T = 210
    q, k, v, dec, want, S = _gla_inputs(T, H, D, Dv, dt, 5, strength)
    pack = torch.zeros((T, sum(-(-x // 8) * 8 for x in (H * D, H * D, H * Dv))), dtype=dt)
    oq, ok, ov = 0, -(-H * D // 8) * 8, 2 * (-(-H * D // 8) * 8)
    pack[:, oq: oq + H * D], pack[:, ok: ok + H * D], pack[:, ov: ov + H * Dv] = q, k, v
    cases = [([T], 1), ([2, 64, 65, 79], 1)]
    if chunked:
        cases += [([T], 2), ([T], 4), ([70, 140], 3)]
    else:
        cases += [([1] * 40 + [T - 40], 1)]
    for cuts, parts in cases:
        state, got, pos = torch.full((3, H, D, Dv), 50.0, device=DEV), [], 0
        for n in cuts:
            x, d = pack[pos: pos + n].to(DEV), dec[pos: pos + n].to(DEV)
            o = torch.zeros((n, H * Dv), dtype=dt, device=DEV)
            M.gla(x[:, oq: oq + H * D], x[:, ok: ok + H * D], x[:, ov: ov + H * Dv], d, o, state, _segs([(0, n, pos, 1)]), q_scale=D ** -0.5,
                  chunked=chunked, parts=parts)
            got.append(o)
            pos += n
        assert _err(torch.cat(got), want) < tol, (cuts, parts)
        assert _err(state[1], S) < (3e-6 if dt == F32 else 1e-4), (cuts, parts)
        assert (state[0] == 50.0).all() and (state[2] == 50.0).all()


def test_gla_many_segments():
    """Segments of unequal lengths in one launch, each as if alone; two that go on and two that start."""
    M = _m()
    H, D, Dv, lens = 2, 48, 72, [100, 17, 64, 130]
    data = [_gla_inputs(n + 30, H, D, Dv, BF, 10 * i, 0.3) for i, n in enumerate(lens)]
    state = torch.full((4, H, D, Dv), 50.0, device=DEV)
    began = [0, 30, 30, 0]
    for i in (1, 2):
        q, k, v, dec = (t[:30].to(DEV).contiguous() for t in data[i][:4])
        pack = torch.cat([q, k, v], 1)
        M.gla(pack[:, : H * D], pack[:, H * D: 2 * H * D], pack[:, 2 * H * D:], dec, torch.zeros((30, H * Dv), dtype=BF, device=DEV), state,
              _segs([(0, 30, 0, i)]), q_scale=D ** -0.5)
    parts = [[t[b: b + n] for t in data[i][:4]] for i, (b, n) in enumerate(zip(began, lens))]
    pack = torch.cat([torch.cat(p[:3], 1) for p in parts]).to(DEV)
    dec = torch.cat([p[3] for p in parts]).to(DEV)
    row0, segs = 0, []
    for i, n in enumerate(lens):
        segs.append((row0, n, began[i], i))
        row0 += n
    o = torch.zeros((row0, H * Dv), dtype=BF, device=DEV)
    M.gla(pack[:, : H * D], pack[:, H * D: 2 * H * D], pack[:, 2 * H * D:], dec, o, state, _segs(segs), q_scale=D ** -0.5, chunked=True, parts=2)
    for (r0, n, b, i) in segs:
        assert _err(o[r0: r0 + n], data[i][4][b: b + n]) < 6e-3


# ---------------------------------------------------------------------------------------------- gated units, logits
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("half", [13, 40, 512])
def test_gated_units(dt, tol, half):
    M = _m()
    g, u = _rand((9, half), 1, dt, 2.0), _rand((9, half), 2, dt, 2.0)
    gd, ud = g.double(), u.double()
    cg, cu = gd.clamp(max=1.2), ud.clamp(-1.2, 1.2)
    kinds = [(M.Glu(0), gd * O.sigmoid(gd) * ud), (M.Glu(1), O.gelu_tanh(gd) * ud),
             (M.Glu(2, 1.2, 1.702, 1.0), cg * O.sigmoid(1.702 * cg) * (cu + 1)), (M.Glu(2, 1.2, 0.5, 0.25), cg * O.sigmoid(0.5 * cg) * (cu + 0.25))]
    turns = torch.stack([g.view(9, -1, 8), u.view(9, -1, 8)], 2).view(9, -1) if half % 8 == 0 else None
    for kind, want in kinds:
        for h, inter in ((torch.cat([g, u], 1), False), (turns, True)):
            if h is None:
                continue
            out = torch.empty((9, half), dtype=dt, device=DEV)
            M.glu(h.to(DEV), out, kind, interleaved=inter)
            assert _err(out, want) < tol, (kind.kind, inter)


def test_scaled_and_capped_logits():
    M = _m()
    x = _rand((5, 40), 1, s=30.0)
    for scale, cap in ((0.3, 7.0), (2.5, 0.0), (1.0, 11.0)):
        got = x.clone().to(DEV)
        M.softcap_(got, 37, cap, scale)
        want = x.double() * scale
        want = cap * torch.tanh(want / cap) if cap else want
        assert _err(got[:, :37], want[:, :37]) < 1e-6 and torch.equal(got[:, 37:].cpu(), x[:, 37:])


# ---------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("n", [1, 5, 200, 300, 1000])
@pytest.mark.parametrize("E,top,groups,keep", [(1, 1, 1, 1), (6, 2, 3, 2), (8, 4, 2, 1), (12, 5, 1, 1), (160, 8, 8, 3), (64, 3, 64, 5)])
def test_gate_route(n, E, top, groups, keep):
    X = _x()
    z, corr = _rand((n, E), 1, s=2.0), _rand((E,), 2, s=0.5) - 1.0        # many choice scores are negative
    cfg = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep} if groups > 1 else None}
    want = O.route(z.double(), corr.double(), cfg)
    wide = torch.full((n, E + 8), 99.0)
    wide[:, :E] = z
    h = _rand((n, 24), 3, BF)
    for align in (1, 32, 128):
        r, by_slot = X.gate_route(wide.to(DEV)[:, :E], corr.to(DEV), top, align, n_groups=groups, keep=keep, h=h.to(DEV) if align == 128 else None)
        slots, rows, start, count, table = (t.cpu() for t in (r.slots, r.rows, r.start, r.count, r.groups))
        owner = torch.full((r.max_slots,), -1)
        for e in range(E):
            assert int(start[e]) % align == 0
            owner[int(start[e]): int(start[e]) + int(count[e])] = e
        assert int(count.sum()) == n * top and len(set(slots.flatten().tolist())) == n * top
        for t in range(n):
            assert sorted(owner[slots[t].long()].tolist()) == sorted(e for e, _ in want[t]), t
            w = dict(want[t])
            for s, got in zip(slots[t].tolist(), r.weight[t].tolist()):
                assert abs(got - float(w[int(owner[s])])) < 1e-5
        assert torch.equal(rows[slots.long()], torch.arange(n, dtype=torch.int32)[:, None].expand(-1, top))
        assert (rows[owner < 0] == -1).all()
        for i in range(r.max_slots // align):
            part = owner[i * align: (i + 1) * align]
            assert int(table[i]) == int(part[0]) and ((part == part[0]) | (part == -1)).all()
        if by_slot is not None:
            assert torch.equal(by_slot[r.slots.long()].cpu(), h[:, None].expand(-1, top, -1))


@pytest.mark.parametrize("n,E,top,W,F,align,dt", [(3, 5, 2, 72, 24, 1, BF), (60, 4, 3, 264, 40, 1, BF), (9, 2, 1, 1104, 16, 1, BF),
                                                  (90, 5, 2, 56, 24, 32, F32), (300, 3, 2, 264, 136, 128, BF), (700, 2, 1, 128, 72, 256, BF)])
def test_gated_experts(n, E, top, W, F, align, dt):
    """Few rows, FP32 and the grouped GEMM on one packing: turns of eight gates and eight values."""
    M, X = _m(), _x()
    h = _rand((n, W), 1, dt)
    gate, up = _rand((E, F, W), 2, dt, W ** -0.5 * 2), _rand((E, F, W), 3, dt, W ** -0.5 * 2)
    both = torch.stack([gate.view(E, -1, 8, W), up.view(E, -1, 8, W)], 2).reshape(E, 2 * F, W).to(DEV)
    r, by_slot = X.gate_route(_rand((n, E), 4).to(DEV), torch.zeros(E, device=DEV), top, align, h=h.to(DEV) if align >= 128 else None)
    got = X.expert_product(h.to(DEV) if by_slot is None else by_slot, both, r, gather=by_slot is None, gate=M.Glu(2, 0.9, 1.702, 1.0))
    owner = torch.zeros(r.max_slots, dtype=torch.long)
    for e in range(E):
        owner[int(r.start[e]): int(r.start[e]) + int(r.count[e])] = e
    live = r.slots.flatten().long().cpu()
    eye = torch.eye(F, dtype=torch.float64)
    for e in range(E):
        mine = live[owner[live] == e]
        if len(mine):
            rows = r.rows.cpu()[mine].long()
            want = O.expert(h[rows].double(), gate[e].double(), up[e].double(), eye, 0.9)
            assert _err(got[mine.to(DEV)], want) < (3e-6 if dt == F32 else 8e-3), e
