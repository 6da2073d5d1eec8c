"""The mixer kernels, each against the plain restatement of its mechanism (float64 on the CPU)."""
import math

import pytest
import torch

from oracles import gugedra as O

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _m():
    from nexus_b200.ops import _mixers as M
    return M


def _segs(parts, width=None):
    """parts: (first row, rows, first position, slot) per segment."""
    M = _m()
    t = torch.zeros((4, width or len(parts)), dtype=torch.int32)
    for i, p in enumerate(parts):
        t[:, i] = torch.tensor(p, dtype=torch.int32)
    return M.Segments(t.to(DEV), 0, len(parts), max(p[1] for p in parts), sum(p[1] for p in parts))


def _rand(shape, seed, dtype=torch.float32, s=1.0):
    x = torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s
    return x.to(dtype)


def _err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).norm() / want.norm().clamp_min(1e-30)).item()


DTYPES = [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)]


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("cols", [96, 50, 2048])
def test_residual_norm(dt, tol, cols):
    M = _m()
    n, ld, eps = 5, (cols + 7) // 8 * 8, 1e-3
    x, y = _rand((n, cols), 1), _rand((n, ld), 2, dt)
    wp, wn = 1 + _rand((cols,), 3, s=0.3), 1 + _rand((cols,), 4, s=0.3)
    xd, h, xc = x.clone().to(DEV), torch.full((n, ld), 7.0, dtype=dt, device=DEV), torch.full((n, ld), 7.0, dtype=dt, device=DEV)
    M.residual_norm(xd, y=y.to(DEV), w_post=wp.to(DEV), w_next=wn.to(DEV), h=h, x_cast=xc, eps=eps)
    want = x.double() + O.rms_norm(y[:, :cols].double(), wp.double(), eps)
    assert _err(xd, want) < 1e-6
    assert _err(h[:, :cols], O.rms_norm(want, wn.double(), eps)) < tol and _err(xc[:, :cols], want) < tol
    assert h[:, cols:].abs().sum() == 0 and xc[:, cols:].abs().sum() == 0
    table, tok = _rand((11, cols), 5, dt), torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32)
    M.residual_norm(xd, tokens=tok.to(DEV), table=table.to(DEV), w_next=wn.to(DEV), h=h, eps=eps)
    assert torch.equal(xd.cpu(), table[tok.long()].float())
    small = torch.full((2, cols), 1e-3)           # eps inside the root matters for a small row
    M.residual_norm(xd[:2].copy_(small), w_next=wn.to(DEV), h=h[:2], eps=eps)
    assert _err(h[:2, :cols], O.rms_norm(small.double(), wn.double(), eps)) < tol


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("dims", [0, 6, 20])
def test_rope_append(dt, tol, dims):
    M = _m()
    H, G, D, Dv, n, bs, base = 6, 2, 20, 12, 9, 4, 300.0
    q_off, k_off, v_off = 8, 8 + 120, 8 + 120 + 40
    ld = v_off + 24 + 5
    proj = _rand((n, ld), 1, dt)
    want = proj.double().clone()
    for off, heads in ((q_off, H), (k_off, G)):
        blk = want[:, off: off + heads * D].reshape(n, heads, D)
        want[:, off: off + heads * D] = O.rotate_half(blk, dims, base).reshape(n, -1) if dims else blk.reshape(n, -1)
    half = dims // 2
    ang = torch.arange(n).double()[:, None] * base ** (-2.0 * torch.arange(half).double() / max(dims, 1))
    kc, vc = torch.zeros((4, bs, G, D), dtype=dt, device=DEV), torch.zeros((4, bs, G, Dv), dtype=dt, device=DEV)
    slots = torch.tensor([12, 13, 14, 15, 0, 1, 2, -1, 4], dtype=torch.int32)
    pd = proj.to(DEV)
    M.rope_append(pd, q_off, k_off, v_off, H, G, D, Dv, dims, torch.arange(n, dtype=torch.int32, device=DEV), slots.to(DEV),
                  ang.cos().float().to(DEV), ang.sin().float().to(DEV), kc, vc)
    assert _err(pd, want) < tol
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(kc.view(-1, G * D)[s].cpu(), pd[r, k_off: k_off + G * D].cpu())
            assert torch.equal(vc.view(-1, G * Dv)[s].cpu(), proj[r, v_off: v_off + G * Dv])
    assert kc.view(-1, G * D)[3].abs().sum() == 0          # the row with a negative slot left nothing behind


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("taps,C", [(1, 10), (2, 33), (3, 64), (4, 130), (8, 24)])
def test_conv_silu_portions(dt, tol, taps, C):
    """Any cutting of a sequence gives what the whole sequence gives; a slot that is used again starts from zeros."""
    M = _m()
    T = 90
    w, b = _rand((C, taps), 2, s=0.5), _rand((C,), 3, s=0.3)
    state = torch.full((3, max(taps - 1, 1), C), 9.0, dtype=dt, device=DEV)
    wd, bd = w.t().contiguous().to(DEV), b.to(DEV)
    for cuts in ([T], [1] * 12 + [T - 12], [2, 3, 33, 1, 1, 50], [32, 32, 26]):
        x, x2 = _rand((T, C), len(cuts), dt), _rand((T, C), 50, dt)
        want = O.silu(O.causal_conv(x.double(), w.double(), b.double()))
        want2 = O.silu(O.causal_conv(x2.double(), w.double()))
        got, got2, pos = [], [], 0
        for n in cuts:
            packed = torch.cat([x[pos: pos + n], torch.zeros(1, C, dtype=dt), x2[pos: pos + n]], 0)
            wide = torch.zeros((2 * n + 1, C + 6), dtype=dt)
            wide[:, 4: 4 + C] = packed
            wide = wide.to(DEV)
            xin = wide[:, 4: 4 + C]
            y = torch.zeros((2 * n + 1, C), dtype=dt, device=DEV)
            M.conv_silu(xin, y, wd, bd, state, _segs([(0, n, pos, 2)]))
            M.conv_silu(xin, y, wd, None, state, _segs([(n + 1, n, pos, 0)]))
            got.append(y[:n])
            got2.append(y[n + 1:])
            pos += n
        assert _err(torch.cat(got), want) < tol and _err(torch.cat(got2), want2) < tol


def _ssd_inputs(T, H, P, N, G, dt, seed):
    xbc = _rand((T, H * P + 2 * G * N), seed, dt)
    raw = _rand((T, H), seed + 1, dt, 2.0)
    dtb, al, D = torch.linspace(-5.0, 1.0, H), torch.linspace(-2.0, 1.5, H), torch.linspace(0.5, 1.5, H)
    x, B, C = xbc.double().split([H * P, G * N, G * N], 1)
    y, S = O.ssd_recurrence(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), O.softplus(raw.double() + dtb), al.double(),
                            D.double())
    return xbc, raw, dtb, al, D, y.reshape(T, H * P), S


SSD_SHAPES = [(3, 16, 24, 3), (4, 56, 40, 2), (2, 20, 10, 1), (4, 72, 136, 2), (2, 64, 128, 1)]


@pytest.mark.parametrize("H,P,N,G", SSD_SHAPES)
@pytest.mark.parametrize("dt,tol,chunked", [(torch.float32, 3e-6, False), (torch.bfloat16, 6e-3, False), (torch.bfloat16, 6e-3, True)])
def test_ssd(H, P, N, G, dt, tol, chunked):
    M = _m()
    T = 210
    xbc, raw, dtb, al, D, want, S = _ssd_inputs(T, H, P, N, G, dt, 5)
    args = [t.to(DEV) for t in (dtb, al, D)]
    cases = [([T], 1), ([2, 64, 65, 79], 1)]
    if chunked:
        cases += [([T], 2), ([T], 4), ([70, 140], 3)]
    else:
        cases += [([1] * 5 + [T - 5], 1)]
    for cuts, parts in cases:
        state = torch.full((4, H, N, P), 3.0, device=DEV)
        y = torch.zeros((T, H * P), dtype=dt, device=DEV)
        pos = 0
        for n in cuts:
            M.ssd(xbc[pos: pos + n].to(DEV), raw[pos: pos + n].to(DEV), y[pos: pos + n], *args, state, G,
                  _segs([(0, n, pos, 1)]), chunked=chunked, parts=parts)
            pos += n
        assert _err(y, want) < tol, (cuts, parts)
        assert _err(state[1], S) < (3e-6 if dt == torch.float32 else 1e-4)      # the state itself is FP32 in both
        assert (state[[0, 2, 3]] == 3.0).all()


def test_ssd_chunk_equals_steps_in_a_batch_of_unequal_segments():
    M = _m()
    H, P, N, G, dt = 4, 48, 40, 2, torch.bfloat16
    lens = [100, 17, 333, 64]
    T = sum(lens)
    xbc, raw, dtb, al, D, _, _ = _ssd_inputs(T, H, P, N, G, dt, 9)
    args = [t.to(DEV) for t in (dtb, al, D)]
    start = _rand((6, H, N, P), 3)
    parts, r = [], 0
    for i, n in enumerate(lens):
        parts.append((r, n, [0, 7, 40, 0][i], [5, 0, 3, 1][i]))
        r += n
    outs = {}
    for mode in ("step", "chunk", "spans"):
        state, y = start.clone().to(DEV), torch.zeros((T, H * P), dtype=dt, device=DEV)
        M.ssd(xbc.to(DEV), raw.to(DEV), y, *args, state, G, _segs(parts), chunked=mode != "step", parts=3 if mode == "spans" else 1)
        outs[mode] = (y.float(), state)
    for mode in ("chunk", "spans"):
        assert _err(outs[mode][0], outs["step"][0]) < 4e-3 and _err(outs[mode][1], outs["step"][1]) < 1e-4
    assert torch.equal(outs["chunk"][1][[2, 4]].cpu(), start[[2, 4]])


def _delta_inputs(T, H, G, D, Dv, dt, seed):
    qkv = _rand((T, 2 * G * D + H * Dv), seed, dt)
    b, a = _rand((T, H), seed + 1, dt, 1.5), _rand((T, H), seed + 2, dt, 1.5)
    al, dtb = torch.linspace(-3.0, 0.5, H), torch.linspace(-4.0, 0.0, H)
    q, k, v = qkv.double().split([G * D, G * D, H * Dv], 1)
    q, k = O.unit(q.reshape(T, G, D)) * D ** -0.5, O.unit(k.reshape(T, G, D))
    g = torch.exp(-torch.exp(al.double()) * O.softplus(a.double() + dtb))
    o, S = O.delta_recurrence(q, k, v.reshape(T, H, Dv), 1 / (1 + torch.exp(-b.double())), g)
    return qkv, b, a, al, dtb, o.reshape(T, H * Dv), S


@pytest.mark.parametrize("H,G,D,Dv", [(3, 3, 32, 48), (6, 2, 24, 40), (2, 1, 20, 10), (2, 2, 128, 64), (2, 1, 136, 72)])
@pytest.mark.parametrize("dt,tol,chunked", [(torch.float32, 3e-6, False), (torch.bfloat16, 6e-3, False), (torch.bfloat16, 6e-3, True)])
def test_delta(H, G, D, Dv, dt, tol, chunked):
    M = _m()
    T = 210
    qkv, b, a, al, dtb, want, S = _delta_inputs(T, H, G, D, Dv, dt, 3)
    for cuts in ([T], [2, 64, 65, 79], [1, 1, 1, 190, 17]):
        state, o, pos = torch.full((3, H, D, Dv), 5.0, device=DEV), torch.zeros((T, H * Dv), dtype=dt, device=DEV), 0
        for n in cuts:
            s = slice(pos, pos + n)
            M.delta(qkv[s].to(DEV), b[s].to(DEV), a[s].to(DEV), o[s], dtb.to(DEV), al.to(DEV), state, G, _segs([(0, n, pos, 2)]),
                    unit_eps=1e-6, q_scale=D ** -0.5, chunked=chunked)
            pos += n
        assert _err(o, want) < tol, cuts
        assert _err(state[2], S) < (3e-6 if dt == torch.float32 else 1e-4)
        assert (state[:2] == 5.0).all()


def test_delta_chunk_with_repeated_keys_and_unit_write_strength():
    """The same key again and again, beta near 1 and no decay: the inverse of the chunk's triangular system has entries far
    from the diagonal that random keys never show."""
    M = _m()
    T, H, G, D, Dv, dt = 130, 2, 1, 32, 16, torch.bfloat16
    qkv, b, a, al, dtb, _, _ = _delta_inputs(T, H, G, D, Dv, dt, 4)
    qkv[:, D: 2 * D] = qkv[:1, D: 2 * D] + 0.3 * qkv[:, D: 2 * D]
    b, a = torch.full_like(b, 4.0), torch.full_like(a, -8.0)
    q, k, v = qkv.double().split([G * D, G * D, H * Dv], 1)
    g = torch.exp(-torch.exp(al.double()) * O.softplus(a.double() + dtb))
    want, S = O.delta_recurrence(O.unit(q.reshape(T, G, D)) * D ** -0.5, O.unit(k.reshape(T, G, D)), v.reshape(T, H, Dv),
                                 1 / (1 + torch.exp(-b.double())), g)
    state, o = torch.zeros((1, H, D, Dv), device=DEV), torch.zeros((T, H * Dv), dtype=dt, device=DEV)
    M.delta(qkv.to(DEV), b.to(DEV), a.to(DEV), o, dtb.to(DEV), al.to(DEV), state, G, _segs([(0, T, 0, 0)]), unit_eps=1e-6,
            q_scale=D ** -0.5, chunked=True)
    assert _err(o, want.reshape(T, -1)) < 6e-3 and _err(state[0], S) < 2e-4


def test_delta_chunk_unit_vectors_of_tiny_inputs():
    """The constant inside the root of the unit vectors decides when q and k are tiny."""
    M = _m()
    T, H, G, D, Dv, dt = 40, 2, 2, 16, 16, torch.bfloat16
    qkv, b, a, al, dtb, _, _ = _delta_inputs(T, H, G, D, Dv, dt, 8)
    qkv[:, : 2 * G * D] *= 2.0 ** -12
    q, k, v = qkv.double().split([G * D, G * D, H * Dv], 1)
    g = torch.exp(-torch.exp(al.double()) * O.softplus(a.double() + dtb))
    want, _ = O.delta_recurrence(O.unit(q.reshape(T, G, D)) * D ** -0.5, O.unit(k.reshape(T, G, D)), v.reshape(T, H, Dv),
                                 1 / (1 + torch.exp(-b.double())), g)
    for chunked in (False, True):
        state, o = torch.zeros((1, H, D, Dv), device=DEV), torch.zeros((T, H * Dv), dtype=dt, device=DEV)
        M.delta(qkv.to(DEV), b.to(DEV), a.to(DEV), o, dtb.to(DEV), al.to(DEV), state, G, _segs([(0, T, 0, 0)]), unit_eps=1e-6,
                q_scale=D ** -0.5, chunked=chunked)
        assert _err(o, want.reshape(T, -1)) < 6e-3


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("groups,size", [(1, 40), (3, 24), (2, 700)])
def test_gated_norm(dt, tol, groups, size):
    M = _m()
    n, eps = 7, 1e-2
    y, z = _rand((n, groups * size), 1, dt), _rand((n, groups * size + 3), 2, dt)
    w, ws = 1 + _rand((groups * size,), 3, s=0.3), 1 + _rand((size,), 4, s=0.3)
    out = torch.zeros((n, groups * size), dtype=dt, device=DEV)
    M.gated_norm(y.to(DEV), z.to(DEV)[:, 3:], w.to(DEV), out, groups=groups, gate_first=True, eps=eps, out_scale=1.7)
    assert _err(out, 1.7 * O.gated_group_norm(y.double(), z[:, 3:].double(), w.double(), groups, eps)) < tol
    M.gated_norm(y.to(DEV), z.to(DEV)[:, 3:], ws.to(DEV), out, groups=groups, gate_first=False, eps=eps)
    want = O.rms_norm(y.double().view(n, groups, size), ws.double(), eps) * O.silu(z[:, 3:].double()).view(n, groups, size)
    assert _err(out, want.view(n, -1)) < tol


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_token_side_silu_mul_softcap(dt, tol):
    M = _m()
    n, dim = 6, 20
    a, table = _rand((n, 24), 1, s=2.0), _rand((9, 3 * dim), 2, dt)
    tok = torch.tensor([8, 0, 3, 3, 1, 5], dtype=torch.int32)
    out = torch.full((n, 24), 5.0, dtype=dt, device=DEV)
    M.token_side_gate(a.to(DEV), tok.to(DEV), table.to(DEV), 2 * dim, out, dim)
    assert _err(out[:, :dim], O.gelu_tanh(a[:, :dim].double()) * table[tok.long(), 2 * dim:].double()) < tol
    assert out[:, dim:].abs().sum() == 0
    for half in (16, 13):
        h, y = _rand((n, 2 * half), 3, dt, 2.0), torch.zeros((n, half), dtype=dt, device=DEV)
        M.silu_mul(h.to(DEV), y)
        assert _err(y, O.silu(h[:, :half].double()) * h[:, half:].double()) < tol
    x = _rand((5, 70), 4, s=20.0)
    xd = x.clone().to(DEV)
    M.softcap_(xd, 66, 7.5)
    assert _err(xd[:, :66], 7.5 * torch.tanh(x[:, :66].double() / 7.5)) < 1e-6 and torch.equal(xd[:, 66:].cpu(), x[:, 66:])


# ------------------------------------------------------------------------------------------------ attention
def _attn_case(T, H, G, D, Dv, dt, seed, hot=()):
    """Random q, k, v; for every (query, key) of ``hot`` the pair points one way, so that its score stands out."""
    q, k, v = _rand((T, H, D), seed), _rand((T, G, D), seed + 1), _rand((T, G, Dv), seed + 2)
    for i, j in hot:
        u = _rand((D,), 100 + j)
        u = u / u.norm()
        q[i] = u * 4.0 * math.sqrt(D)
        k[j] = u * 3.0
    return q.to(dt), k.to(dt), v.to(dt)


def _run_paged(q, k, v, segs, table, cache_rows, bs, window, scale, cap, splits, out_scale):
    """segs: (first row, rows, first position, slot); cache_rows: slot -> tokens of that sequence already known (k, v)."""
    M = _m()
    G, D, Dv = k[0].shape[1], k[0].shape[2], v[0].shape[2]
    dt = q.dtype
    nb = int(table.max()) + 1
    kc, vc = torch.full((nb * bs, G, D), 50.0, dtype=dt), torch.full((nb * bs, G, Dv), 50.0, dtype=dt)
    for s, n in cache_rows.items():
        p = torch.arange(n)
        slot = table[s][p // bs].long() * bs + p % bs
        kc[slot], vc[slot] = k[s][:n], v[s][:n]
    H = q.shape[1]
    out = torch.zeros((q.shape[0], H * Dv + 4), dtype=dt, device=DEV)
    single = [s for s in segs if s[1] == 1]
    many = [s for s in segs if s[1] > 1]
    for part in (single, many) if dt == torch.bfloat16 else (segs,):
        if part:
            M.paged_window_attention(q.reshape(q.shape[0], -1).to(DEV), kc.view(nb, bs, G, D).to(DEV), vc.view(nb, bs, G, Dv).to(DEV),
                                     table.to(DEV), out[:, 4:], _segs(part), heads=H, block_size=bs, window=window, scale=scale,
                                     softcap=cap, out_scale=out_scale, splits=splits)
    return out[:, 4:].float().cpu()


@pytest.mark.parametrize("H,G,D,Dv", [(12, 2, 64, 64), (4, 2, 32, 24), (3, 3, 20, 48), (6, 2, 80, 128), (20, 1, 16, 16), (2, 1, 192, 256),
                                      (5, 1, 12, 9)])
@pytest.mark.parametrize("dt,tol", [(torch.float32, 3e-6), (torch.bfloat16, 8e-3)])
def test_paged_window_attention(H, G, D, Dv, dt, tol):
    """Prompts, portions and single tokens of three sequences over scattered pages; queries whose best key is the last one
    inside the window, the first one outside it, or sits on a page border."""
    bs, window, scale, cap = 16, 45, 0.7 / math.sqrt(D), 6.0
    lens = {0: 150, 2: 90, 3: 33}
    hot = {0: [(149, 149 - window + 1), (148, 148 - window), (130, 112), (131, 95)], 2: [(89, 89 - window + 1), (60, 48), (61, 47)],
           3: [(32, 0), (20, 16)]}
    data = {s: _attn_case(n, H, G, D, Dv, dt, 10 + s, hot[s]) for s, n in lens.items()}
    table = torch.randperm(60, generator=torch.Generator().manual_seed(1))[:48].view(4, 12).to(torch.int32)
    want = {s: O.window_attention(*[t.double() for t in data[s]], scale, cap, window) for s in lens}
    k, v = {s: d[1] for s, d in data.items()}, {s: d[2] for s, d in data.items()}
    kl, vl = [k.get(s, k[0]) for s in range(4)], [v.get(s, v[0]) for s in range(4)]
    for cut, splits in (({0: 0, 2: 0, 3: 0}, 1), ({0: 101, 2: 88, 3: 31}, 1), ({0: 149, 2: 89, 3: 32}, 1), ({0: 149, 2: 60, 3: 32}, 3)):
        rows, segs, r = [], [], 0
        for s in (2, 0, 3):
            n = lens[s] - cut[s]
            rows.append(data[s][0][cut[s]:])
            segs.append((r, n, cut[s], s))
            r += n
        got = _run_paged(torch.cat(rows), kl, vl, segs, table, lens, bs, window, scale, cap, splits, 0.6)
        ref = torch.cat([want[s][cut[s]:] for s in (2, 0, 3)]).reshape(r, -1) * 0.6
        assert _err(got, ref) < tol, (cut, splits)
        worst = ((got.double() - ref).norm(dim=1) / ref.norm(dim=1)).max().item()
        assert worst < 4 * tol, (cut, worst)


@pytest.mark.parametrize("window,cap", [(0, 0.0), (1, 3.0), (64, 0.0), (500, 9.0)])
def test_paged_window_attention_other_masks(window, cap):
    H, G, D, Dv, T, bs = 4, 2, 32, 32, 140, 16
    table = torch.arange(12, dtype=torch.int32).flip(0).view(1, 12)
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        q, k, v = _attn_case(T, H, G, D, Dv, dt, 3)
        qd, kd, vd = q.double(), k.double(), v.double()
        want = O.window_attention(qd, kd, vd, 0.3, cap if cap else 1e9, window if window else 10 ** 6)
        got = _run_paged(q, [k], [v], [(0, T, 0, 0)], table, {0: T}, bs, window, 0.3, cap, 1, 1.0)
        assert _err(got, want.reshape(T, -1)) < tol
        got = _run_paged(q[-1:], [k], [v], [(0, 1, T - 1, 0)], table, {0: T}, bs, window, 0.3, cap, 4, 1.0)
        assert _err(got, want[-1].reshape(1, -1)) < tol


def test_flash_attention_window_softcap_and_output_scale():
    """The tcgen05 kernel that fresh prompts take: window edge, soft cap and output factor against the restatement."""
    from nexus_b200.ops import _cuda as K
    T, H, G, D, window, cap = 200, 4, 1, 64, 70, 8.0
    hot = [(199, 130), (198, 128), (150, 81), (128, 58)]
    q, k, v = _attn_case(T, H, G, D, D, torch.bfloat16, 7, hot)
    want = O.window_attention(q.double(), k.double(), v.double(), 0.09, cap, window).reshape(T, -1) * 0.6
    got, _ = K.attention_fwd(q[None].to(DEV), k[None].to(DEV), v[None].to(DEV), causal=True, window=window, scale=0.09, softcap=cap,
                             out_scale=0.6)
    got = got[0].reshape(T, -1).float().cpu()
    assert _err(got, want) < 8e-3 and ((got.double() - want).norm(dim=1) / want.norm(dim=1)).max() < 3e-2
    K.check_status()
