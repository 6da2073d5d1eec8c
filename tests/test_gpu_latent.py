"""The kernels of latent attention and of table-routed experts, each against the plain restatement of its mechanism."""
import math

import pytest
import torch

from oracles import makuzen as O

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)]


def _m():
    from nexus_b200.ops import _mixers as M
    return M


def _x():
    from nexus_b200.ops import _experts as X
    return X


def _rand(shape, seed, dtype=torch.float32, s=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s).to(dtype)


def _err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).norm() / want.norm().clamp_min(1e-30)).item()


def _segs(parts):
    """parts: (first row, rows, first position, slot) per segment."""
    t = torch.tensor(parts, dtype=torch.int32).t().contiguous()
    return _m().Segments(t.to(DEV), 0, len(parts), max(p[1] for p in parts), sum(p[1] for p in parts))


def _tables(rot, n):
    freq, mul = O.yarn_frequencies(rot["dims"], rot["base"], rot["scaling"])
    ang = torch.arange(n).double()[:, None] * torch.tensor(freq, dtype=torch.float64)
    return (ang.cos() * mul).float().to(DEV), (ang.sin() * mul).float().to(DEV)


ROT = {"base": 300.0, "scaling": {"factor": 4.0, "original": 40, "fast": 6.0, "slow": 0.5}}


# ---------------------------------------------------------------------------------------------- norms, rotation, residual
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,dims,H", [(44, 56, 16, 5), (21, 37, 6, 17), (192, 512, 64, 16)])
def test_latent_prep(dt, tol, q_rank, kv_rank, dims, H):
    M = _m()
    n, bs, eps = 9, 8, 1e-3
    rot_col, row = -(-kv_rank // 16) * 16, -(-(kv_rank + 16 + dims) // 64) * 64
    off, at = [], 3 if q_rank == 21 else 8
    for size in (q_rank, kv_rank, dims, H):
        off.append(at)
        at += -(-size // 8) * 8
    proj = _rand((n, at + 5 - at % 2 if q_rank == 21 else at), 1, dt)
    wq, wk = 1 + _rand((q_rank,), 2, s=0.3), 1 + _rand((kv_rank,), 3, s=0.3)
    pos = torch.tensor([0, 1, 2, 3, 40, 41, 90, 5, 7], dtype=torch.int32)
    slots = torch.tensor([12, 13, 14, 15, 0, 1, 2, -1, 4], dtype=torch.int32)
    rot = {"dims": dims, **ROT}
    cos, sin = _tables(rot, 100)
    cq = torch.full((n, -(-q_rank // 8) * 8), 7.0, dtype=dt, device=DEV)
    cache = torch.zeros((2, bs, 1, row), dtype=dt, device=DEV)
    lat = torch.full((n, row), 7.0, dtype=dt, device=DEV)
    gate = torch.zeros((n, H), device=DEV)
    M.latent_prep(proj.to(DEV), off, q_rank, kv_rank, dims, H, wq.to(DEV), wk.to(DEV), pos.to(DEV), slots.to(DEV), cos, sin, cq, cache,
                  rot_col, gate, eps=eps, lat=lat)
    p = proj.double()
    assert _err(cq[:, :q_rank], O.rms_norm(p[:, off[0]: off[0] + q_rank], wq.double(), eps)) < tol and cq[:, q_rank:].abs().sum() == 0
    c = O.rms_norm(p[:, off[1]: off[1] + kv_rank], wk.double(), eps)
    full = torch.zeros((100, 1, dims), dtype=torch.float64)
    kr = torch.stack([O.rotate(full.index_fill(0, pos[r].long(), 0).index_copy(0, pos[r: r + 1].long(), p[r: r + 1, None, off[2]: off[2] + dims]),
                               rot)[pos[r], 0] for r in range(n)])
    assert _err(lat[:, :kv_rank], c) < tol and _err(lat[:, rot_col: rot_col + dims], kr) < tol
    assert lat[:, kv_rank:rot_col].abs().sum() == 0 and lat[:, rot_col + dims:].abs().sum() == 0
    assert _err(gate, O.sigmoid(p[:, off[3]: off[3] + H])) < 1e-5
    rows = cache.view(-1, row)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(rows[s], lat[r])
    assert rows[3].abs().sum() == 0                      # the row with a negative slot left nothing behind


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("dims,width,H", [(6, 16, 3), (32, 32, 6), (64, 128, 16)])
def test_rope_heads(dt, tol, dims, width, H):
    M = _m()
    n, own = 23, 24
    rot = {"dims": dims, **ROT}
    cos, sin = _tables(rot, n)
    src = _rand((n, H * (own + dims)), 1, dt)
    want = O.rotate(src.double().view(n, H, -1)[:, :, own:], rot)
    dst = torch.full((n, H * (40 + width)), 7.0, dtype=dt, device=DEV)
    pos = torch.arange(n, dtype=torch.int32, device=DEV)
    s = src.to(DEV)
    M.rope_heads(s, own + dims, own, dst, 40 + width, 40, H, dims, width, pos, cos, sin)
    got = dst.view(n, H, -1)
    assert _err(got[:, :, 40: 40 + dims], want) < tol and got[:, :, 40 + dims:].abs().sum() == 0 and (got[:, :, :40] == 7).all()
    M.rope_heads(s, own + dims, own, s, own + dims, own, H, dims, dims, pos, cos, sin)      # in place
    assert _err(s.view(n, H, -1)[:, :, own:], want) < tol and torch.equal(s.view(n, H, -1)[:, :, :own].cpu(), src.view(n, H, -1)[:, :, :own])


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("cols,top", [(88, 2), (50, 3), (2048, 1)])
def test_residual_norm_with_experts(dt, tol, cols, top):
    M = _m()
    n, ld, eps, slots_n = 6, -(-cols // 8) * 8, 1e-3, 40
    g = torch.Generator().manual_seed(0)
    slots = torch.randperm(slots_n, generator=g)[: n * top].view(n, top).to(torch.int32)
    x, y, ex = _rand((n, cols), 1), _rand((n, ld), 2, dt), _rand((slots_n, ld), 3, dt)
    w, dot, gate = 1 + _rand((cols,), 4, s=0.3), _rand((cols,), 5, s=cols ** -0.5), torch.rand(n, generator=g)
    xd, xc = x.clone().to(DEV), torch.full((n, ld), 7.0, dtype=dt, device=DEV)
    sg, by_slot = torch.zeros(n, device=DEV), torch.full((slots_n, ld), 7.0, dtype=dt, device=DEV)
    M.residual_norm(xd, y=y.to(DEV), w_post=w.to(DEV), x_cast=xc, eps=eps, res_mult=0.3, experts=ex.to(DEV), slots=slots.to(DEV), top=top,
                    y_gate=gate.to(DEV), w_dot=dot.to(DEV), dot_out=sg, scatter=by_slot)
    mean = ex.double()[slots.long(), :cols].mean(1)
    want = x.double() + 0.3 * O.rms_norm(mean + gate.double()[:, None] * y.double()[:, :cols], w.double(), eps)
    assert _err(xd, want) < 1e-6 and _err(xc[:, :cols], want) < tol and xc[:, cols:].abs().sum() == 0
    assert _err(sg, O.sigmoid(want @ dot.double())) < 1e-5
    for r in range(n):
        for s in slots[r].tolist():
            assert torch.equal(by_slot[s], xc[r])
    rest = sorted(set(range(slots_n)) - set(slots.flatten().tolist()))
    assert (by_slot[rest] == 7).all()
    M.residual_norm(xd, w_post=w.to(DEV), eps=eps, experts=ex.to(DEV), slots=slots.to(DEV), top=top)      # no shared expert
    assert _err(xd, want + O.rms_norm(mean, w.double(), eps)) < 1e-5
    table, tok = _rand((11, cols), 5, dt), torch.tensor([3, 10, 0, 3, 7, 1], dtype=torch.int32)
    M.residual_norm(xd, tokens=tok.to(DEV), table=table.to(DEV), x_cast=xc, eps=eps, embed_scale=2.5)
    assert torch.equal(xd.cpu(), table[tok.long()].float() * 2.5)


# ---------------------------------------------------------------------------------------------- experts
def _skewed(n, experts, top, seed):
    """Experts of every token, most of them the same few; expert 1 is never used when there is room."""
    g = torch.Generator().manual_seed(seed)
    p = torch.rand((n, experts), generator=g) * (torch.arange(experts, 0, -1).float() ** 2)
    if experts > top + 1:
        p[:, 1] = -1
    return p.topk(top, -1).indices.to(torch.int32)


@pytest.mark.parametrize("align", [1, 32, 128])
def test_table_route(align):
    X = _x()
    vocab, n = 61, 300
    tokens = torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(1), dtype=torch.int32)
    shapes = [(6, 2), (1, 1), (40, 5), (1100, 3)] + [(9, 1)] * 35                 # more layers than one launch takes
    layers = [(_skewed(vocab, e, top, i), e) for i, (e, top) in enumerate(shapes)]
    routes = X.table_route(tokens.to(DEV), [(t.to(DEV), e) for t, e in layers], align)
    for (table, experts), r in zip(layers, routes):
        want = table[tokens.long()]
        slots, rows, start, count, groups = (t.cpu().long() for t in (r.slots, r.rows, r.start, r.count, r.groups))
        assert torch.equal(count, want.flatten().long().bincount(minlength=experts))
        assert (start % align == 0).all() and len(set(slots.flatten().tolist())) == slots.numel()
        assert torch.equal(rows[slots], torch.arange(n)[:, None].expand_as(slots))
        assert ((slots >= start[want.long()]) & (slots < start[want.long()] + count[want.long()])).all()
        used = torch.full_like(groups, -1)
        for e in range(experts):
            used[int(start[e]) // align: (int(start[e]) + int(count[e]) + align - 1) // align] = e
        assert torch.equal(groups, used) and (rows >= 0).sum() == slots.numel()


@pytest.mark.parametrize("align,dt", [(1, torch.bfloat16), (128, torch.bfloat16), (256, torch.bfloat16), (32, torch.float32)])
@pytest.mark.parametrize("n,E,top,k,ff", [(5, 3, 2, 56, 24), (70, 9, 4, 320, 72), (333, 4, 1, 1152, 264), (640, 5, 3, 128, 512)])
def test_expert_products(align, dt, n, E, top, k, ff):
    """Up with squared relu, then down, for skewed counts (an unused expert, one with most rows)."""
    X = _x()
    tokens = torch.arange(n, dtype=torch.int32)
    table = _skewed(n, E, top, n)
    r = X.table_route(tokens.to(DEV), [(table.to(DEV), E)], align)[0]
    h, up, down = _rand((n, k), 1, dt), _rand((E, ff, k), 2, dt, k ** -0.5), _rand((E, k, ff), 3, dt, ff ** -0.5)
    by_slot = h[r.rows.cpu().long().clamp_min(0)].to(DEV)
    gather = align < 128
    a = X.expert_product(h.to(DEV) if gather else by_slot, up.to(DEV), r, gather=gather, act="relu2")
    y = X.expert_product(a, down.to(DEV), r, gather=False)
    slots = r.slots.cpu().long()
    mid = torch.stack([torch.stack([O.squared_relu(up[e].double() @ h[t].double()) for e in table[t].long().tolist()]) for t in range(n)])
    tol = 2e-6 if dt == torch.float32 else 6e-3
    assert _err(a.cpu()[slots], mid) < tol
    got = a.cpu()[slots].double()                       # the second product from the first one's rounded output
    want = torch.stack([torch.stack([down[e].double() @ got[t, j] for j, e in enumerate(table[t].long().tolist())]) for t in range(n)])
    assert _err(y.cpu()[slots], want) < tol


def test_grouped_gemm_skips_and_large_tiles():
    from nexus_b200.ops import _cuda as K
    g = torch.Generator().manual_seed(0)
    a, b = torch.randn(1024, 200, generator=g).bfloat16(), torch.randn(3, 520, 200, generator=g).bfloat16()
    for rows in (128, 256):
        groups = torch.tensor([2, -1, 0, 0, 1, -1, 2, -1][: 1024 // rows], dtype=torch.int32)
        out = torch.full((1024, 520), 3.0, dtype=torch.bfloat16, device=DEV)
        K.grouped_gemm(a.to(DEV), b.to(DEV), groups.to(DEV), rows, out=out)
        K.check_status()
        for i, e in enumerate(groups.tolist()):
            part = out[i * rows: (i + 1) * rows].cpu()
            if e < 0:
                assert (part == 3).all()
            else:
                assert _err(part, a[i * rows: (i + 1) * rows].double() @ b[e].double().t()) < 6e-3
    with pytest.raises(ValueError):
        K.grouped_gemm(a.to(DEV), b.to(DEV), groups[:2].to(DEV), 128)


@pytest.mark.parametrize("m,n,k,split", [(7, 72, 64, 1), (100, 300, 1024, 4), (300, 512, 256, 1), (300, 96, 256, 1)])
def test_squared_relu_epilogues(m, n, k, split):
    from nexus_b200.ops import _cuda as K
    from nexus_b200.ops import _infer as I
    x, w = _rand((m, k), 1, torch.bfloat16), _rand((n, k), 2, torch.bfloat16, k ** -0.5)
    want = O.squared_relu(x.double() @ w.double().t())
    assert _err(K.gemm(x.to(DEV), w.to(DEV), act="relu2", split_k=split, deterministic=True), want) < 6e-3
    if m <= 16:
        assert _err(I.skinny_gemm(x.to(DEV), w.to(DEV), act="relu2"), want) < 6e-3


@pytest.mark.parametrize("n,H,k,N", [(1, 3, 48, 16), (13, 5, 128, 512), (70, 2, 512, 128), (250, 4, 64, 40)])
def test_head_product(n, H, k, N):
    X = _x()
    x, w = _rand((n, H, k + 24), 1, torch.bfloat16), _rand((H, N, k), 2, torch.bfloat16, k ** -0.5)
    out = torch.full((n, H, N + 8), 7.0, dtype=torch.bfloat16, device=DEV)
    X.head_product(x.to(DEV)[:, :, :k], w.to(DEV), out[:, :, :N])
    assert _err(out[:, :, :N], torch.einsum("nhk,hmk->nhm", x[:, :, :k].double(), w.double())) < 6e-3 and (out[:, :, N:] == 7).all()


# ---------------------------------------------------------------------------------------------- attention over the latent cache
def _paged(lengths, bs, row, rank, seed, dt):
    """Latent rows of sequences of the given lengths in shuffled pages; the other slots hold large values."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // bs) for n in lengths]
    pages = torch.randperm(sum(per) + 3, generator=g)
    cache = torch.full((len(pages), bs, 1, row), 300.0, dtype=dt)
    table = torch.zeros((len(lengths), max(per) + 1), dtype=torch.int32)
    lat, p = [], 0
    for i, n in enumerate(lengths):
        c = torch.randn(n, row, generator=g).to(dt)
        lat.append(c)
        for b in range(per[i]):
            table[i, b] = pages[p]
            part = c[b * bs: (b + 1) * bs]
            cache[pages[p], : len(part), 0] = part
            p += 1
    return cache, table, lat


def _absorbed_ref(q, lat, segs, H, rank, window, scale, gate):
    out = torch.zeros((q.shape[0], H, rank), dtype=torch.float64)
    for r0, n, p0, seq in segs:
        c = lat[seq][: p0 + n].double()
        qq = torch.zeros((p0 + n, H, c.shape[1]), dtype=torch.float64)
        qq[p0:] = q[r0: r0 + n].double().view(n, H, -1)
        for i in range(p0, p0 + n):
            lo = max(0, i - window + 1) if window else 0
            s = (qq[i] @ c[lo: i + 1].t()) * scale
            out[r0 + i - p0] = torch.softmax(s, -1) @ c[lo: i + 1, :rank]
    return (out * gate.double()[:, :, None]).view(q.shape[0], -1)


ABSORBED = [(6, 96, 32, 16), (16, 512, 64, 16), (5, 48, 16, 24), (20, 256, 48, 8), (70, 112, 16, 32), (1, 16, 16, 64), (32, 512, 64, 16),
            (24, 512, 200, 16)]


@pytest.mark.parametrize("window", [0, 1, 33, 130])
@pytest.mark.parametrize("H,rank,rot,bs", ABSORBED)
def test_latent_attention(H, rank, rot, bs, window):
    """Decoding and portions over shuffled pages, with and without spans of the keys."""
    M = _m()
    row, lengths = -(-(rank + rot) // 64) * 64, [150, 1, 64, 65]
    cache, table, lat = _paged(lengths, bs, row, rank, H, torch.bfloat16)
    cache[..., rank + rot:] = 0
    lat = [c.clone() for c in lat]
    for c in lat:
        c[:, rank + rot:] = 0
    scale = (rank + rot) ** -0.5
    for segs in ([(0, 1, 149, 0), (2, 1, 0, 1), (1, 1, 63, 2), (3, 1, 64, 3)], [(0, 13, 137, 0), (14, 2, 0, 2), (16, 60, 5, 3)]):
        n = max(s[0] + s[1] for s in segs)
        q, gate = _rand((n, H * row), 7, torch.bfloat16), torch.rand((n, H), generator=torch.Generator().manual_seed(3))
        want = _absorbed_ref(q, lat, segs, H, rank, window, scale, gate)
        live = torch.tensor(sorted(r for s in segs for r in range(s[0], s[0] + s[1])))
        for splits in (1, 3):
            out = torch.full((n, H * rank), 7.0, dtype=torch.bfloat16, device=DEV)
            M.latent_attention(q.to(DEV), cache.to(DEV), table.to(DEV), out, _segs(segs), heads=H, rank=rank, window=window, scale=scale,
                               gate=gate.to(DEV), splits=splits)
            assert _err(out[live.to(DEV)], want[live]) < 6e-3, (segs, splits)
    from nexus_b200.ops import _cuda as K
    K.check_status()


def test_latent_attention_finds_one_key_at_every_edge():
    """One key answers a query far above all others: its latent is the output while the window holds it, and not one token
    later; also with a large negative scale in front of a reversed query."""
    M = _m()
    H, rank, rot, bs, row, T = 3, 48, 16, 16, 64, 200
    cache, table, lat = _paged([T], bs, row, rank, 1, torch.bfloat16)
    for sign in (1.0, -1.0):
        for window in (0, 17, 64, 100):
            for key in (0, 15, 16, 31, 32, 99, 150):
                poss = [p for p in {key, key + 1, (key + window - 1) if window else T - 1, key + window, T - 1} if key <= p < T]
                q = torch.stack([lat[0][key].float() * 4 * sign for _ in poss]).bfloat16().repeat(1, H)
                segs = [(i, 1, p, 0) for i, p in enumerate(poss)]
                gate = torch.ones((len(poss), H), device=DEV)
                for splits in (1, 4):
                    out = torch.zeros((len(poss), H * rank), dtype=torch.bfloat16, device=DEV)
                    M.latent_attention(q.to(DEV), cache.to(DEV), table.to(DEV), out, _segs(segs), heads=H, rank=rank, window=window,
                                       scale=sign, gate=gate, splits=splits)
                    for i, p in enumerate(poss):
                        hit = _err(out[i].view(H, rank), lat[0][key, :rank].expand(H, -1)) < 1e-2
                        assert hit == (window == 0 or p - key < window), (window, key, p)


@pytest.mark.parametrize("H,rank,rot,window", [(5, 56, 16, 19), (17, 512, 64, 0), (2, 1024, 32, 40)])
def test_fp32_latent_attention(H, rank, rot, window):
    M = _m()
    row, segs = -(-(rank + rot) // 64) * 64, [(0, 1, 70, 0), (1, 25, 6, 1)]
    cache, table, lat = _paged([71, 31], 8, row, rank, 2, torch.float32)
    n = 26
    q, gate = _rand((n, H * row), 7), torch.rand((n, H), generator=torch.Generator().manual_seed(3))
    out = torch.zeros((n, H * rank), device=DEV)
    M.paged_window_attention(q.to(DEV), cache.to(DEV), None, table.to(DEV), out, _segs(segs), heads=H, block_size=8, window=window,
                             scale=0.05, gate=gate.to(DEV), vdim=rank)
    assert _err(out, _absorbed_ref(q, lat, segs, H, rank, window, 0.05, gate)) < 5e-6


@pytest.mark.parametrize("window", [0, 40])
def test_paged_window_kernels_on_a_latent_cache(window):
    """The general BF16 kernels: values as the leading columns of the keys, gated outputs, spans of the keys."""
    M = _m()
    H, rank, row = 5, 96, 128
    cache, table, lat = _paged([150, 60], 16, row, rank, 2, torch.bfloat16)
    for segs, splits in (([(0, 1, 149, 0), (1, 1, 59, 1)], 1), ([(0, 1, 149, 0), (1, 1, 59, 1)], 3), ([(0, 70, 80, 0), (70, 30, 10, 1)], 1)):
        n = max(s[0] + s[1] for s in segs)
        q, gate = _rand((n, H * row), 7, torch.bfloat16), torch.rand((n, H), generator=torch.Generator().manual_seed(3))
        out = torch.zeros((n, H * rank), dtype=torch.bfloat16, device=DEV)
        M.paged_window_attention(q.to(DEV), cache.to(DEV), None, table.to(DEV), out, _segs(segs), heads=H, block_size=16, window=window,
                                 scale=0.08, gate=gate.to(DEV), vdim=rank, splits=splits)
        assert _err(out, _absorbed_ref(q, lat, segs, H, rank, window, 0.08, gate)) < 6e-3


# ---------------------------------------------------------------------------------------------- attention of prompts
def _prompt_ref(q, kv, lat, segs, H, dim, rot, vdim, rank, window, scale, gate):
    out = torch.zeros((q.shape[0], H, vdim), dtype=torch.float64)
    for r0, n, p0, kv0 in segs:
        L = p0 + n
        k = torch.cat([kv[kv0: kv0 + L, : H * dim].double().view(L, H, dim), lat[kv0: kv0 + L, None, rank: rank + rot].double().expand(L, H, rot)], -1)
        v = kv[kv0: kv0 + L, H * dim:].double().view(L, H, vdim)
        s = torch.einsum("thd,khd->htk", q[r0: r0 + n].double().view(n, H, dim + rot), k) * scale
        i, j = torch.arange(p0, L)[:, None], torch.arange(L)[None]
        see = (j <= i) & (j > i - window) if window else j <= i
        out[r0: r0 + n] = torch.einsum("htk,khd->thd", s.masked_fill(~see, float("-inf")).softmax(-1), v)
    return (out * gate.double()[:, :, None]).view(q.shape[0], -1)


def _blocks(segs, window):
    from nexus_b200.infer.prompt import long_segments
    out = []
    for r0, n, p0, kv0 in segs:
        for b in long_segments([(r0, n, 0, 0)], window)[0]:
            out.append([b[0], b[1], p0 + b[2], kv0])
    return torch.tensor(out, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("window", [0, 1, 40, 129, 300])
@pytest.mark.parametrize("dim,rot,vdim,H", [(128, 64, 128, 3), (64, 32, 64, 6), (16, 16, 8, 5), (96, 48, 72, 2), (32, 64, 128, 2)])
def test_latent_prompt(dim, rot, vdim, H, window):
    """Segments of many lengths, some of them behind earlier tokens, packed beside one another."""
    M = _m()
    segs = [(0, 20, 0, 0), (20, 300, 0, 20), (320, 513, 100, 320), (833, 128, 7, 940), (961, 129, 0, 1080)]
    n, kv_n, rank = 1090, 1209, 48
    q, kv, lat = _rand((n, H * (dim + rot)), 1, torch.bfloat16), _rand((kv_n, H * (dim + vdim)), 2, torch.bfloat16), _rand((kv_n, 128), 3, torch.bfloat16)
    gate, scale = torch.rand((n, H), generator=torch.Generator().manual_seed(3)), (dim + rot) ** -0.5
    out = torch.full((n, H * vdim), 7.0, dtype=torch.bfloat16, device=DEV)
    M.latent_prompt(q.to(DEV), kv.to(DEV), lat.to(DEV), out, _blocks(segs, window), heads=H, dim=dim, rot=rot, vdim=vdim, rank=rank,
                    window=window, scale=scale, gate=gate.to(DEV))
    from nexus_b200.ops import _cuda as K
    K.check_status()
    assert _err(out, _prompt_ref(q, kv, lat, segs, H, dim, rot, vdim, rank, window, scale, gate)) < 6e-3


def test_latent_prompt_finds_one_key_at_every_edge():
    """Every query asks for the key a fixed distance back, once through its own part, once through the shared part."""
    M = _m()
    H, dim, rot, vdim, rank, n = 2, 64, 32, 64, 16, 520
    unit = torch.nn.functional.normalize(_rand((n, H * (dim + vdim)), 2).view(n, -1, 32), dim=-1) * 32 ** 0.5    # keys of one length
    kv, lat = unit.view(n, -1).bfloat16(), (torch.nn.functional.normalize(_rand((n, 2, 32), 3), dim=-1) * 32 ** 0.5).roll(rank, -1)
    lat = torch.cat([torch.zeros(n, rank), lat[:, 0], torch.zeros(n, 64 - rank - rot)], 1).bfloat16()
    v = kv[:, H * dim:].view(n, H, vdim)
    for window in (1, 64, 100, 129, 256):
        for back in {0, 1, window - 1, window}:
            for shared in (False, True):
                q = torch.zeros((n, H, dim + rot))
                src = torch.arange(n) - back
                ok = src >= 0
                if shared:
                    q[ok, :, dim:] = lat[src[ok], None, rank: rank + rot].float() * 4
                else:
                    q[ok, :, :dim] = kv[src[ok], : H * dim].view(-1, H, dim).float() * 4
                out = torch.zeros((n, H * vdim), dtype=torch.bfloat16, device=DEV)
                M.latent_prompt(q.bfloat16().view(n, -1).to(DEV), kv.to(DEV), lat.to(DEV), out, _blocks([(0, n, 0, 0)], window), heads=H,
                                dim=dim, rot=rot, vdim=vdim, rank=rank, window=window, scale=1.0)
                d = (out.float().cpu().view(n, H, vdim)[ok] - v[src[ok]].float()).flatten(1).norm(dim=1) / v[src[ok]].float().flatten(1).norm(dim=1)
                assert (d < 2e-2).all() if back < window else (d > 0.1).all(), (window, back, shared)


def test_latent_gather():
    M = _m()
    cache, table, lat = _paged([150, 40], 24, 128, 64, 5, torch.bfloat16)
    runs = torch.tensor([[0, 100, 50, 0], [100, 40, 0, 1]], dtype=torch.int32, device=DEV)
    dst = torch.zeros((140, 128), dtype=torch.bfloat16, device=DEV)
    M.latent_gather(cache.to(DEV), table.to(DEV), runs, 100, dst)
    assert torch.equal(dst.cpu(), torch.cat([lat[0][50:150], lat[1]]))


def test_kernels_refuse_bad_arguments():
    from nexus_b200.ops import _cuda as K
    M = _m()
    cache, table, _ = _paged([20], 8, 64, 48, 0, torch.bfloat16)
    q, out = torch.zeros((1, 2 * 64), dtype=torch.bfloat16, device=DEV), torch.zeros((1, 2 * 48), dtype=torch.bfloat16, device=DEV)
    with pytest.raises(RuntimeError):
        M.latent_attention(q, cache.to(DEV), table.to(DEV), out, _segs([(0, 1, 3, 0)]), heads=2, rank=600, window=0, scale=1.0)
    with pytest.raises(RuntimeError):
        M.latent_prompt(q, q, q, out, torch.zeros((1, 4), dtype=torch.int32, device=DEV), heads=1, dim=16, rot=16, vdim=8, rank=0, window=0,
                        scale=-1.0)
    K.check_status()
    assert math.isfinite(float(out.float().sum()))
