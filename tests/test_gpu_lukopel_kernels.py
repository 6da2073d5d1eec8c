"""The kernels of residual streams, normed heads, chunked and biased attention and heads that mix their weights, each against the plain
restatement of its mechanism."""
import pytest
import torch

from oracles import lukopel as O

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
DTYPES = [(F32, 3e-6), (BF, 6e-3)]


def _m():
    from nexus_b200.ops import _mixers as M
    return M


def _rand(shape, seed, dtype=F32, s=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s).to(dtype)


def _err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).norm() / want.norm().clamp_min(1e-30)).item()


def _rows_err(got, want):
    """The worst row."""
    got, want = got.double().cpu().flatten(1), want.double().cpu().flatten(1)
    return ((got - want).norm(dim=1) / want.norm(dim=1).clamp_min(1e-30)).max().item()


def _segs(parts, max_len=0):
    """parts: (first row, rows, first position, slot) per segment."""
    t = torch.tensor(parts, dtype=torch.int32).t().contiguous()
    return _m().Segments(t.to(DEV), 0, len(parts), max_len or max(p[1] for p in parts), sum(p[1] for p in parts))


# ---------------------------------------------------------------------------------------------- residual
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("streams,cols", [(1, 96), (2, 50), (3, 2048), (4, 88), (5, 40), (8, 24), (7, 4096), (2, 12288), (1, 20480), (4, 3001)])
def test_residual_streams(dt, tol, streams, cols):
    M = _m()
    n, V, P, ld, eps = 7, 30, 40, (cols + 7) // 8 * 8, 1e-3
    table, pos_table = _rand((V, cols), 1, dt), _rand((P, cols), 2, dt)
    tok, pos = torch.tensor([3, 29, 0, 3, 7, 8, 9], dtype=torch.int32), torch.tensor([0, 39, 5, 17, 2, 2, 1], dtype=torch.int32)
    read, w = _rand((streams,), 3), 1 + _rand((cols,), 4, s=0.3)
    x = torch.full((n, streams, cols), 9.0, device=DEV)
    h = torch.full((n, ld), 9.0, dtype=dt, device=DEV)
    M.stream_residual(x, tokens=tok.to(DEV), table=table.to(DEV), embed_scale=2.5, positions=pos.to(DEV), pos_table=pos_table.to(DEV),
                      read=read.to(DEV), w_next=w.to(DEV), h=h, eps=eps)
    e = table[tok.long()].double() * 2.5 + pos_table[pos.long()].double()
    xs = e.repeat(streams, 1, 1)
    assert _err(x.transpose(0, 1), xs) < 1e-6
    assert _err(h[:, :cols], O.norm(sum(read[s].double() * xs[s] for s in range(streams)), w.double(), eps)) < tol
    assert (h[:, cols:] == 0).all()
    # a sublayer's output joins, the next one's input leaves; every stream from the old ones
    x0, y = _rand((n, streams, cols), 5), _rand((n, ld), 6, dt)
    p = {"in": _rand((streams,), 7).double(), "out": _rand((streams,), 8).double(), "mix": _rand((streams, streams), 9).double()}
    want = O.hyper_step(x0.transpose(0, 1).double(), p, lambda u: y[:, :cols].double())
    x = x0.to(DEV)
    dev = {k: v.float().to(DEV) for k, v in p.items()}
    M.stream_residual(x, y=y.to(DEV), mix=dev["mix"], out=dev["out"], read=read.to(DEV), w_next=w.to(DEV), h=h, eps=eps)
    assert _err(x.transpose(0, 1), want) < 1e-6
    assert _err(h[:, :cols], O.norm(sum(read[s].double() * want[s] for s in range(streams)), w.double(), eps)) < tol
    # without a next sublayer; then the sum of the streams, which nothing else changes
    x = x0.to(DEV)
    M.stream_residual(x, y=y.to(DEV), mix=dev["mix"], out=dev["out"], eps=eps)
    assert _err(x.transpose(0, 1), want) < 1e-6
    M.stream_residual(x, w_next=w.to(DEV), h=h, eps=eps)
    assert _err(x.transpose(0, 1), want) < 1e-6 and _err(h[:, :cols], O.norm(want.sum(0), w.double(), eps)) < tol


@pytest.mark.parametrize("dt,tol", DTYPES)
def test_learned_positions_of_one_stream(dt, tol):
    M = _m()
    table, pos_table, w = _rand((9, 52), 1, dt), _rand((12, 52), 2, dt), 1 + _rand((52,), 3, s=0.2)
    tok, pos = torch.tensor([8, 0, 3], dtype=torch.int32), torch.tensor([11, 0, 4], dtype=torch.int32)
    x, h = torch.empty((3, 52), device=DEV), torch.empty((3, 56), dtype=dt, device=DEV)
    M.residual_norm(x, tokens=tok.to(DEV), table=table.to(DEV), eps=1e-4, embed_scale=0.5, positions=pos.to(DEV), pos_table=pos_table.to(DEV),
                    w_next=w.to(DEV), h=h)
    want = table[tok.long()].double() * 0.5 + pos_table[pos.long()].double()
    assert _err(x, want) < 1e-6 and _err(h[:, :52], O.norm(want, w.double(), 1e-4)) < tol


# ---------------------------------------------------------------------------------------------- heads
@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,pad", [(6, 2, 24, 20, True), (4, 4, 64, 64, False), (3, 1, 7, 5, True), (32, 8, 128, 64, False)])
@pytest.mark.parametrize("whole", [False, True])
def test_head_prep(dt, tol, heads, kv, dim, vdim, pad, whole):
    M = _m()
    n, slots, eps = 9, 40, 1e-2
    D, Dv = ((dim + 15) // 16 * 16, (vdim + 7) // 8 * 8) if pad else (dim, vdim)
    q, k, v, g = _rand((n, heads * dim), 1, dt), _rand((n, kv * dim), 2, dt), _rand((n, kv * vdim), 3, dt), _rand((n, heads), 4, dt)
    wq, wk = 1 + _rand((heads * dim if whole else dim,), 5, s=0.3), 1 + _rand((kv * dim if whole else dim,), 6, s=0.3)
    per_head = 1 + _rand((heads,), 7, s=0.5)
    pos, slot = torch.tensor([0, 1, 21, 22, 23, 45, 46, 900, 3], dtype=torch.int32), torch.tensor([5, 39, 0, 7, -1, 8, 9, 30, 31], dtype=torch.int32)
    coef, every, scale = 0.4, 23, -0.2

    def padded(t, heads, size):
        out = torch.zeros(t.shape[0], heads, size, dtype=t.dtype)
        out[:, :, : t.shape[1] // heads] = t.view(t.shape[0], heads, -1)
        return out.flatten(1)

    def weight(t, heads):
        return padded(t[None], heads if whole else 1, D)[0].to(DEV)
    proj = torch.cat([padded(q, heads, D), padded(k, kv, D), padded(v, kv, Dv), padded(g, 1, (heads + 7) // 8 * 8)], 1).to(DEV)
    at = (0, heads * D, (heads + kv) * D, (heads + kv) * D + kv * Dv)
    norm = O.whole_norm if whole else O.head_norm
    want_q = norm(q.double(), wq.double(), heads, eps) * scale * per_head.double()[None, :, None]
    want_q = want_q * torch.tensor([1 + coef * torch.log(torch.tensor((int(p) + 1) // every + 1.0, dtype=torch.float64)) for p in pos])[:, None, None]
    want_k = norm(k.double(), wk.double(), kv, eps)
    plain_v = v.double().view(n, kv, vdim)
    for unit, store in ((True, True), (False, False)):
        kc, vc = torch.full((slots, kv, D), 7.0, dtype=dt, device=DEV), torch.full((slots, kv, Dv), 7.0, dtype=dt, device=DEV)
        gate, x = torch.empty((n, heads), device=DEV), proj.clone()
        M.head_prep(x, at, heads=heads, kv_heads=kv, dim=D, vdim=Dv, norm_dim=dim, norm_vdim=vdim, eps=eps, w_q=weight(wq, heads),
                    w_k=weight(wk, kv), positions=pos.to(DEV), slots=slot.to(DEV), k_cache=kc, v_cache=vc, norm_all=whole, unit_values=unit,
                    store_kv=store, q_scale=scale, head_scale=per_head.to(DEV), coef=coef, every=every, gate=gate)
        want_v = O.rms(plain_v, eps) if unit else plain_v
        assert _err(x[:, : at[1]].view(n, heads, D)[:, :, :dim], want_q) < tol
        assert _err(gate, torch.sigmoid(g.double())) < 1e-6
        ok = slot >= 0
        assert _err(kc[slot[ok].long().to(DEV)][:, :, :dim], want_k[ok]) < tol and _err(vc[slot[ok].long().to(DEV)][:, :, :vdim], want_v[ok]) < tol
        if store:
            assert _err(x[:, at[1]: at[2]].view(n, kv, D)[:, :, :dim], want_k) < tol
            assert _err(x[:, at[2]: at[3]].view(n, kv, Dv)[:, :, :vdim], want_v) < tol
        else:
            assert torch.equal(x[:, at[1]:], proj[:, at[1]:])
        untouched = torch.ones(slots, dtype=torch.bool)
        untouched[slot[ok].long()] = False
        assert (kc[untouched.to(DEV)] == 7).all() and (vc[untouched.to(DEV)] == 7).all()
        assert (kc[:, :, dim:][~untouched.to(DEV)] == 0).all()


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("heads,kv,vdim", [(6, 3, 24), (4, 1, 20), (32, 8, 64), (9, 1, 128), (24, 2, 40), (5, 5, 13)])
def test_head_mix(dt, tol, heads, kv, vdim):
    M = _m()
    n = 11
    wide, talk, gate = _rand((n, heads, kv, vdim), 1, dt), _rand((heads, heads), 2), torch.rand((n, heads), generator=torch.Generator().manual_seed(3))
    for g in (gate, None):
        out = torch.empty((n, heads * vdim), dtype=dt, device=DEV)
        M.head_mix(wide.to(DEV).view(n, -1), talk.to(DEV), None if g is None else g.to(DEV), out, heads=heads, kv_heads=kv, vdim=vdim)
        all_values = torch.einsum("hg,ngcd->nhcd", talk.double(), wide.double())
        want = all_values[:, torch.arange(heads), torch.arange(heads) // (heads // kv)]
        want = want if g is None else want * g.double()[:, :, None]
        assert _err(out.view(n, heads, vdim), want) < tol


# ---------------------------------------------------------------------------------------------- attention
def _visible(first, n, window, chunk):
    """[n, first + n] of the rows at positions first .."""
    T = first + n
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = O.same_chunk(T, chunk) if chunk else O.causal(T)
    if window:
        see = see & (i - j < window)
    return see[first:]


def _weights(q, k, first, window, chunk, bias, scale):
    """Softmax weights [H, n, first + n] of rows at positions first .. against all keys."""
    H, n, T = q.shape[1], q.shape[0], k.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, O.grouped(k, H)) * scale
    if bias is not None:
        dist = (torch.arange(first, T)[:, None] - torch.arange(T)[None, :]).clamp(0, bias.shape[1] - 1)
        s = s + bias[:, dist]
    return O.weights_of(s, _visible(first, n, window, chunk))


class Case:
    """Sequences in a paged cache with permuted pages; ``stand_out``: positions whose keys every query scores high (whoever sees one of
    them sees little else)."""

    def __init__(self, dt, heads, kv, dim, vdim, lens, firsts, bias_len=0, bs=16, seed=0, stand_out=(), scale=0.3):
        self.dt, self.H, self.G, self.D, self.Dv, self.bs, self.scale = dt, heads, kv, dim, vdim, bs, scale
        g = torch.Generator().manual_seed(seed)
        self.lens, self.firsts = lens, firsts
        self.bias = torch.randn((heads, bias_len), generator=g) if bias_len else None
        self.blocks = max(-(-(f + n) // bs) for f, n in zip(firsts, lens)) + 1
        order = torch.randperm(len(lens) * self.blocks + 3, generator=g)
        self.table = order[: len(lens) * self.blocks].view(len(lens), -1).to(torch.int32)
        self.kc, self.vc = (torch.randn((order.numel(), bs, kv, d), generator=g).to(dt) for d in (dim, vdim))
        self.q, self.k, self.v = [], [], []
        for s, (f, n) in enumerate(zip(firsts, lens)):
            q, k, v = (torch.randn((m, h, d), generator=g) for m, h, d in ((n, heads, dim), (f + n, kv, dim), (f + n, kv, vdim)))
            q[:, :, 0] = 4.0
            k[:, :, 0] = 0.0
            for j in stand_out:
                if j < f + n:
                    k[j, :, 0] = 9.0
            self.q.append(q.to(dt)), self.k.append(k.to(dt)), self.v.append(v.to(dt))
            for j in range(f + n):
                b = self.table[s, j // bs]
                self.kc[b, j % bs], self.vc[b, j % bs] = self.k[-1][j], self.v[-1][j]
        rows, parts = 0, []
        for s, (f, n) in enumerate(zip(firsts, lens)):
            parts.append((rows, n, f, s))
            rows += n
        self.rows, self.parts = rows, parts
        self.qd = torch.cat(self.q).view(rows, -1).to(DEV)

    def args(self):
        return self.kc.to(DEV), self.vc.to(DEV), self.table.to(DEV)

    def bias_d(self):
        return None if self.bias is None else self.bias.to(DEV)

    def weights(self, s, window, chunk):
        return _weights(self.q[s].double(), self.k[s].double(), self.firsts[s], window, chunk, None if self.bias is None else self.bias.double(),
                        self.scale)

    def want(self, window=0, chunk=0, talk=None, gate=None):
        """[rows, H, Dv]"""
        out = []
        for s in range(len(self.lens)):
            p = self.weights(s, window, chunk)
            if talk is not None:
                p = torch.einsum("hg,gij->hij", talk.double(), p)
            out.append(torch.einsum("hij,jhd->ihd", p, O.grouped(self.v[s].double(), self.H)))
        out = torch.cat(out)
        return out if gate is None else out * gate.double()[:, :, None]

    def want_all(self, window=0, chunk=0):
        """[rows, H, G, Dv]: every head's weights with the values of every KV head"""
        return torch.cat([torch.einsum("hij,jgd->ihgd", self.weights(s, window, chunk), self.v[s].double()) for s in range(len(self.lens))])


SIZES = [(6, 2, 24, 20), (4, 4, 64, 64), (5, 1, 16, 136), (8, 2, 128, 64), (34, 2, 40, 24)]


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim", SIZES)
@pytest.mark.parametrize("window,chunk,bias_len", [(0, 21, 0), (0, 0, 37), (30, 48, 9), (0, 200, 300), (0, 1, 0)])
def test_paged_attention_with_chunks_and_biases(dt, tol, heads, kv, dim, vdim, window, chunk, bias_len):
    M = _m()
    gate = torch.rand((400, heads), generator=torch.Generator().manual_seed(9))
    for lens, firsts in (([1, 1, 1, 1], [0, 20, 41, 300]), ([2, 17, 70, 3], [19, 0, 33, 250])):
        c = Case(dt, heads, kv, dim, vdim, lens, firsts, bias_len)
        seg = _segs(c.parts)
        kw = dict(heads=heads, block_size=c.bs, window=window, chunk=chunk, scale=c.scale, bias=c.bias_d())
        for splits in (1, 3) if lens[0] == 1 else (1,):
            out = torch.empty((c.rows, heads * vdim), dtype=dt, device=DEV)
            M.paged_window_attention(c.qd, *c.args(), out, seg, gate=gate[: c.rows].to(DEV), splits=splits, **kw)
            assert _rows_err(out, c.want(window, chunk, gate=gate[: c.rows])) < 3 * tol
        if lens[0] > 1 or dt == F32:
            wide = torch.empty((c.rows, heads * kv * vdim), dtype=dt, device=DEV)
            M.paged_window_attention(c.qd, *c.args(), wide, seg, all_values=True, **kw)
            assert _rows_err(wide, c.want_all(window, chunk)) < 3 * tol


@pytest.mark.parametrize("dt,tol", DTYPES)
@pytest.mark.parametrize("key", [0, 15, 16, 31, 32, 63, 64, 95, 96])
def test_a_key_that_stands_out_at_every_edge(dt, tol, key):
    """Chunks of 32 and of 48 over pages of 16: the rows on both sides of the key's chunk, in prompts, short segments and decoding."""
    M = _m()
    for chunk in (32, 48, 64):
        for lens, firsts in (([130, 9], [0, 90]), ([7, 2], [60, 94]), ([1] * 5, [31, 32, 47, 48, 96])):
            c = Case(dt, 4, 2, 32, 32, lens, firsts, 0, stand_out=(key,))
            out = torch.empty((c.rows, 4 * 32), dtype=dt, device=DEV)
            M.paged_window_attention(c.qd, *c.args(), out, _segs(c.parts), heads=4, block_size=16, window=0, chunk=chunk, scale=c.scale)
            assert _rows_err(out, c.want(0, chunk)) < 3 * tol


@pytest.mark.parametrize("heads,kv,dim,vdim", SIZES)
@pytest.mark.parametrize("window,chunk,bias_len", [(0, 0, 37), (30, 0, 0), (0, 21, 300)])
def test_heads_that_mix_on_short_segments(heads, kv, dim, vdim, window, chunk, bias_len, monkeypatch):
    M = _m()
    talk = 0.5 * torch.eye(heads) + _rand((heads, heads), 4, s=0.5)
    gate = torch.rand((400, heads), generator=torch.Generator().manual_seed(9))
    for lens, firsts in (([1, 1, 1, 1], [0, 63, 64, 300]), ([2, 16, 7, 3, 1], [19, 0, 130, 250, 64])):
        c = Case(BF, heads, kv, dim, vdim, lens, firsts, bias_len)
        kw = dict(heads=heads, block_size=c.bs, window=window, chunk=chunk, scale=c.scale, bias=c.bias_d(), keys=320)
        want = c.want(window, chunk, talk, gate[: c.rows])
        for splits, scratch in ((1, 1 << 29), (3, 1 << 29), (2, 1)):          # the last one: a launch per segment
            monkeypatch.setattr(M, "TALK_SCRATCH", scratch)
            out = torch.full((c.rows + 1, heads * vdim), 5.0, dtype=BF, device=DEV)
            # a segment without rows, as in a captured batch
            M.talk_paged(c.qd, *c.args(), out[: c.rows], talk.to(DEV), _segs([*c.parts, (c.rows, 0, 0, 0)], max(lens)), splits=splits,
                         gate=gate[: c.rows].to(DEV), **kw)
            got = out[: c.rows].view(want.shape)
            assert _rows_err(got, want) < 2.5e-2 and _err(got, want) < 8e-3 and (out[c.rows:] == 5).all()


@pytest.mark.parametrize("key", [0, 15, 16, 36, 37, 63, 64, 127, 128])
def test_heads_that_mix_a_key_that_stands_out(key):
    """Only one head scores the key high, and other heads take its weight over: a mixture before the softmax, a head that is left out or a
    transposed mixture shows."""
    M = _m()
    talk = torch.eye(4) * 0.3
    talk[2, 0], talk[1, 3], talk[0, 0] = 1.0, -0.7, 0.0
    for lens, firsts in (([1, 1, 1], [key, 130, 200]), ([5, 2], [max(0, key - 2), 129])):
        c = Case(BF, 4, 2, 32, 32, lens, firsts, 40, stand_out=(key,))
        for q in c.q:
            q[:, 1:, 0] = 0
        c.qd = torch.cat(c.q).view(c.rows, -1).to(DEV)
        out = torch.empty((c.rows, 4 * 32), dtype=BF, device=DEV)
        M.talk_paged(c.qd, *c.args(), out, talk.to(DEV), _segs(c.parts), heads=4, block_size=16, window=0, scale=c.scale, keys=256,
                     bias=c.bias_d())
        assert _rows_err(out, c.want(talk=talk)) < 2.5e-2


# ---------------------------------------------------------------------------------------------- prompts on tcgen05
def _prompt(c, window, chunk, gathered):
    """Query rows, keys and values, and the blocks of the sequences of a case."""
    from nexus_b200.infer.prompt import long_segments
    blocks, runs, kv_rows = long_segments(c.parts, window, 0, chunk)
    assert bool(runs) == gathered
    if gathered:
        k, v = torch.zeros((kv_rows, c.G, c.D), dtype=BF), torch.zeros((kv_rows, c.G, c.Dv), dtype=BF)
        for first, n, pos, seq in runs:
            k[first: first + n], v[first: first + n] = c.k[seq][pos: pos + n], c.v[seq][pos: pos + n]
    else:
        k, v = torch.cat(c.k), torch.cat(c.v)
    return k.flatten(1).to(DEV), v.flatten(1).to(DEV), torch.tensor([b[:4] for b in blocks], dtype=torch.int32, device=DEV)


PROMPTS = [([17, 300, 129], [0, 0, 0]), ([290, 20, 140], [37, 0, 505])]
PROMPT_SIZES = [(4, 2, 48, 64), (6, 3, 128, 128), (5, 5, 16, 24), (3, 1, 80, 72), (16, 8, 64, 64), (10, 5, 32, 96)]


@pytest.mark.parametrize("heads,kv,dim,vdim", PROMPT_SIZES)
@pytest.mark.parametrize("window,chunk,bias_len", [(0, 0, 121), (0, 50, 0), (0, 256, 700), (37, 0, 9), (0, 300, 33), (0, 0, 1)])
def test_prompts(heads, kv, dim, vdim, window, chunk, bias_len):
    """Fresh prompts and portions behind cached keys: attention with chunks, biases and gates, and every head's weights with the values
    of every KV head."""
    from nexus_b200.ops import _cuda as K
    M = _m()
    for lens, firsts in PROMPTS:
        c = Case(BF, heads, kv, dim, vdim, lens, firsts, bias_len, stand_out=(49, 50, 255, 256, 299, 300), scale=1.0)
        for q in c.q:
            q.mul_(0.3)
        c.qd = torch.cat(c.q).view(c.rows, -1).to(DEV)
        k, v, blocks = _prompt(c, window, chunk, firsts[0] > 0)
        gate = torch.rand((c.rows, heads), generator=torch.Generator().manual_seed(9))
        kw = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, window=window, chunk=chunk, scale=1.0)
        out = torch.empty((c.rows, heads * vdim), dtype=BF, device=DEV)
        M.window_prompt(c.qd, k, v, out, blocks, gate=gate.to(DEV), bias=c.bias_d(), **kw)
        assert _rows_err(out, c.want(window, chunk, gate=gate)) < 1.5e-2
        wide = torch.empty((c.rows, heads * kv * vdim), dtype=BF, device=DEV)
        ext = None if c.bias is None else M.extended_bias(c.bias_d())
        M.talk_prompt(c.qd, k, v, wide, blocks, bias=ext, distances=bias_len, **kw)
        K.check_status()
        assert _rows_err(wide, c.want_all(window, chunk)) < 1.5e-2
        # the mixture, in slices of two or three blocks
        from nexus_b200.infer.prompt import row_slices
        talk = 0.5 * torch.eye(heads) + _rand((heads, heads), 4, s=0.5)
        slices = [(torch.tensor(b, dtype=torch.int32, device=DEV), r, n) for b, r, n in row_slices(blocks.tolist(), 300)]
        assert len(slices) > 1
        M.talk_prompt_mixed(c.qd, k, v, out, slices, talk.to(DEV), gate.to(DEV), bias=ext, distances=bias_len, **kw)
        assert _rows_err(out, c.want(window, chunk, talk, gate)) < 4e-2
        again = torch.empty_like(wide)
        for _ in range(5):
            M.talk_prompt(c.qd, k, v, again, blocks, bias=ext, distances=bias_len, **kw)
            assert torch.equal(again, wide)


def test_prompts_with_growing_scores():
    """Row maxima that keep growing from tile to tile, so that the output tile is rescaled again and again by either softmax group."""
    from nexus_b200.ops import _cuda as K
    M = _m()
    for step in (0.02, 0.4, 1.0):
        c = Case(BF, 4, 2, 32, 64, [700], [0], 50, scale=1.0)
        c.q[0][:, :, 0] = 1.0
        c.k[0][:, :, 0] = (torch.arange(700) * step)[:, None].to(BF)
        c.qd = c.q[0].view(700, -1).to(DEV)
        k, v, blocks = _prompt(c, 0, 0, False)
        wide = torch.empty((700, 4 * 2 * 64), dtype=BF, device=DEV)
        M.talk_prompt(c.qd, k, v, wide, blocks, heads=4, kv_heads=2, dim=32, vdim=64, window=0, scale=1.0,
                      bias=M.extended_bias(c.bias_d()), distances=50)
        K.check_status()
        assert _rows_err(wide, c.want_all()) < 1.5e-2


def test_refused_arguments():
    """What the host checks turn down is never launched."""
    M = _m()
    c = Case(BF, 4, 2, 32, 32, [1], [3])
    out = torch.empty((1, 4 * 32), dtype=BF, device=DEV)
    with pytest.raises(RuntimeError):
        M.paged_window_attention(c.qd, *c.args(), out, _segs(c.parts), heads=4, block_size=16, window=0, chunk=-1, scale=1.0)
    k, v, blocks = _prompt(c, 0, 0, True)
    wide = torch.empty((1, 4 * 2 * 32), dtype=BF, device=DEV)
    with pytest.raises(RuntimeError):
        M.talk_prompt(c.qd, k, v, wide, blocks, heads=4, kv_heads=2, dim=32, vdim=32, window=0, scale=-1.0)
    with pytest.raises(RuntimeError):
        M.stream_residual(torch.zeros((1, 9, 16), device=DEV), w_next=torch.ones(16, device=DEV), h=torch.zeros((1, 16), device=DEV), eps=1e-5)
