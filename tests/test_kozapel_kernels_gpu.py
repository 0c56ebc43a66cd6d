"""Kozapel's mechanisms one by one, each through the C ABI against a plain reference of the same equation: residual streams, gated gelu and
squared-relu matmuls, routing by corrected sigmoids, differential attention (masks, far keys, key splits, shared keys, gate), latent
attention with a query latent and without a window."""
import numpy as np
import pytest
import torch

from gptrs_b200 import model as gm
from gptrs_b200 import ops
from oracle import kozapel_ref as kr

pytestmark = pytest.mark.gpu


def _dev(a, cuda, dt=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).to(cuda)
    return t if dt is None else t.to(dt)


def _i32(a, cuda):
    return torch.tensor(list(a), dtype=torch.int32, device=cuda)


def _f32(rng, *shape):
    return rng.standard_normal(shape).astype(np.float32)


# ---- residual streams --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("dim", [24, 37, 512, 700, 2048, 3072, 5001])
def test_stream_step(cuda, streams, dim):
    rng = np.random.default_rng(dim + streams)
    n = 13
    x, y = _f32(rng, n, streams, dim), 3 * _f32(rng, n, dim)
    mix, w_out, w_in, g = _f32(rng, streams, streams), _f32(rng, streams), _f32(rng, streams), 1 + 0.3 * _f32(rng, dim)
    want = kr.stream_update(x.transpose(1, 0, 2).astype(float), y.astype(float), mix.astype(float), w_out.astype(float))
    want_h = kr.rms(kr.stream_input(want, w_in.astype(float)), 1e-4) * g
    kw = dict(mix=_dev(mix, cuda), w_out=_dev(w_out, cuda))
    gx = _dev(x, cuda)
    h, total = ops.stream_step(gx, 1e-4, y=_dev(y, cuda), w_in=_dev(w_in, cuda), gamma_in=_dev(g, cuda), want_sum=True, **kw)
    assert np.abs(gx.cpu().numpy().transpose(1, 0, 2) - want).max() < 5e-5
    assert np.abs(h.cpu().numpy() - want_h).max() < 1e-4 and np.abs(total.cpu().numpy() - want.sum(axis=0)).max() < 1e-4
    gx = _dev(x, cuda)
    assert ops.stream_step(gx, 1e-4, y=_dev(y, cuda), **kw) == (None, None)   # nothing follows
    assert np.abs(gx.cpu().numpy().transpose(1, 0, 2) - want).max() < 5e-5
    # the end of the model: the sum of the streams, gathered rows, bf16 with padding columns; x is left alone
    yb, ldh, rows = kr.to_bf16(y), (dim + 7) // 8 * 8, [12, 0, 0, 7]
    gx = _dev(x, cuda)
    h, _ = ops.stream_step(gx, 1e-4, y=_dev(yb, cuda, torch.bfloat16), gamma_in=_dev(g, cuda), rows=_i32(rows, cuda), out_dtype=torch.bfloat16, ldh=ldh, **kw)
    last = kr.stream_update(x.transpose(1, 0, 2).astype(float), yb.astype(float), mix.astype(float), w_out.astype(float)).sum(axis=0)
    ref = (kr.rms(last, 1e-4) * g)[rows]
    assert np.abs(h[:, :dim].float().cpu().numpy() - ref).max() < 2 ** -8 * np.abs(ref).max() and (h[:, dim:] == 0).all()
    assert np.array_equal(gx.cpu().numpy(), x)
    h, _ = ops.stream_step(gx, 1e-4, w_in=_dev(w_in, cuda), gamma_in=_dev(g, cuda))   # no sublayer output
    assert np.abs(h.cpu().numpy() - kr.rms(kr.stream_input(x.transpose(1, 0, 2).astype(float), w_in.astype(float)), 1e-4) * g).max() < 1e-4
    assert np.array_equal(gx.cpu().numpy(), x)
    # without weights: the ordinary residual in every stream
    h, _ = ops.stream_step(gx, 1e-4, y=_dev(y, cuda), gamma_in=_dev(g, cuda))
    plain = x + y[:, None]
    assert np.abs(gx.cpu().numpy() - plain).max() < 1e-5 and np.abs(h.cpu().numpy() - kr.rms(plain.sum(axis=1).astype(float), 1e-4) * g).max() < 1e-4


@pytest.mark.parametrize("streams,dim", [(3, 72), (6, 72), (2, 45)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_stream_step_sums_the_experts(cuda, streams, dim, dt):
    rng = np.random.default_rng(0)
    n, top = 11, 3
    x, y, extra = _f32(rng, n, streams, dim), kr.to_bf16(_f32(rng, n * top, dim)), kr.to_bf16(_f32(rng, n, dim))
    mix, w_out, g = _f32(rng, streams, streams), _f32(rng, streams), 1 + 0.3 * _f32(rng, dim)
    pair, w = rng.permutation(n * top).reshape(n, top), rng.random((n, top)).astype(np.float32)
    for add in (False, True):
        out = np.einsum("nk,nkd->nd", w.astype(float), y[pair].astype(float)) + (extra if add else 0)
        want = kr.stream_update(x.transpose(1, 0, 2).astype(float), out, mix.astype(float), w_out.astype(float))
        gx = _dev(x, cuda)
        h, _ = ops.stream_step(gx, 1e-5, y=_dev(y, cuda, dt), mix=_dev(mix, cuda), w_out=_dev(w_out, cuda), gamma_in=_dev(g, cuda), pair=_dev(pair.astype(np.int32), cuda),
                               pair_weight=_dev(w, cuda), add=_dev(extra, cuda, dt) if add else None)
        assert np.abs(gx.cpu().numpy().transpose(1, 0, 2) - want).max() < 5e-5
        assert np.abs(h.cpu().numpy() - kr.rms(want.sum(axis=0), 1e-5) * g).max() < 1e-4


@pytest.mark.parametrize("streams,d", [(3, 44), (7, 44), (1, 21)])
def test_stream_step_embedding(cuda, streams, d):
    rng = np.random.default_rng(1)
    v, n = 30, 25
    table, g, w_in = _f32(rng, v, d), _f32(rng, d), _f32(rng, streams)
    tok = rng.integers(0, v, n)
    x = torch.full((n, streams, d), 9.0, device=cuda)
    kw = dict(embed=_dev(table, cuda), embed_scale=6.5, w_in=_dev(w_in, cuda), gamma_in=_dev(g, cuda))
    h, _ = ops.stream_step(x, 1e-6, tokens=_i32(tok, cuda), **kw)
    want = kr.embed(tok, table.astype(float), 6.5)
    assert np.abs(x.cpu().numpy() - want[:, None]).max() < 1e-5 and np.abs(h.cpu().numpy() - kr.rms(want * w_in.sum(), 1e-6) * g).max() < 5e-5
    for t in (v, -1):   # out of range: flagged, nothing read outside the table
        status = torch.zeros(1, dtype=torch.int32, device=cuda)
        tok[4] = t
        ops.stream_step(x, 1e-6, tokens=_i32(tok, cuda), status=status, **kw)
        assert int(status) == 2


# ---- matmuls with the activations --------------------------------------------------------------------------------------
def _interleave(gate, up):
    """[F][W] each -> [2 F'][W], 8 gates, then their 8 partners; F' = F rounded up to 8."""
    f, w = gate.shape
    fp = (f + 7) // 8 * 8
    out = np.zeros((fp // 8, 2, 8, w), np.float32)
    for part, a in enumerate((gate, up)):
        padded = np.zeros((fp, w), np.float32)
        padded[:f] = a
        out[:, part] = padded.reshape(fp // 8, 8, w)
    return out.reshape(2 * fp, w)


@pytest.mark.parametrize("m,f,w", [(1, 8, 8), (3, 37, 40), (16, 136, 72), (33, 20, 136), (64, 512, 320), (100, 72, 64), (129, 40, 24), (300, 200, 200), (1500, 1544, 256)])
def test_gated_gelu(cuda, m, f, w):
    """From -12 to 12 standard deviations, so that the tails of the tanh are there too; silu beside it."""
    rng = np.random.default_rng(m + f)
    gate, up = (kr.to_bf16((_f32(rng, f, w) * s / w ** 0.5).astype(np.float32)) for s in (4.0, 1.0))
    x = kr.to_bf16(_f32(rng, m, w))
    fp = (f + 7) // 8 * 8
    both = _interleave(gate, up)
    z = x.astype(float) @ gate.T.astype(float)
    for kind, act in ((ops.GATE_GELU_TANH, kr.gelu_tanh), (ops.GATE_SILU, lambda t: t * kr.sigmoid(t))):
        want = act(z) * (x.astype(float) @ up.T.astype(float))
        got = ops.dense_bf16(_dev(x, cuda, torch.bfloat16), _dev(both, cuda, torch.bfloat16), m, 2 * fp, w, swiglu=kind).float().cpu().numpy()
        assert np.abs(got[:, :f] - want).max() < 2 ** -8 * np.abs(want).max() + 1e-3 and (got[:, f:] == 0).all()
        pairs = ops.dense_f32(_dev(x, cuda), _dev(both.T, cuda), m, 2 * fp, w)
        got = ops.gated_pairs_f32(pairs, fp, kind).cpu().numpy()
        assert np.abs(got[:, :f] - want).max() < 1e-5 * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (20, 264, 136), (64, 136, 512), (128, 72, 40), (129, 40, 24), (700, 264, 328)])
def test_squared_relu(cuda, m, n, k):
    rng = np.random.default_rng(m)
    x, w = kr.to_bf16(_f32(rng, m, k)), kr.to_bf16((_f32(rng, n, k) / k ** 0.5).astype(np.float32))
    want = kr.relu2(x.astype(float) @ w.T.astype(float))
    got = ops.dense_bf16(_dev(x, cuda, torch.bfloat16), _dev(w, cuda, torch.bfloat16), m, n, k, relu2=True).float().cpu().numpy()
    assert np.abs(got - want).max() < 2 ** -8 * np.abs(want).max()
    got = ops.dense_f32(_dev(x, cuda), _dev(w.T, cuda), m, n, k, relu2=True).cpu().numpy()
    assert np.abs(got - want).max() < 1e-5 * max(1.0, want.max())


# ---- experts -----------------------------------------------------------------------------------------------------------
ROUTES = [(1, 4, 2, 2, 1), (5, 12, 3, 4, 2), (64, 64, 4, 8, 3), (128, 33, 5, 3, 2), (129, 6, 6, 2, 2), (300, 8, 2, 8, 3), (300, 1, 1, 1, 1), (700, 96, 2, 6, 1),
          (900, 512, 8, 16, 4), (37, 1024, 40, 1, 1), (50, 300, 7, 100, 9)]


@pytest.mark.parametrize("rows,experts,top,groups,keep", ROUTES)
def test_route_by_corrected_sigmoids(cuda, rows, experts, top, groups, keep):
    """Groups that are out hold better choices than some that are chosen, corrections change the choice and make scores negative."""
    rng = np.random.default_rng(rows + experts)
    z, h = 2 * _f32(rng, rows, experts), _f32(rng, rows, 20)
    corr = rng.uniform(-1.5, 0.3, experts).astype(np.float32)
    for tile in (8, 128):
        pair, weight, tiles, n_tiles, out, most = ops.moe_route(experts, top, groups, keep, tile, _dev(z, cuda), _dev(h, cuda), sigmoid=True, group_best=2, weight_scale=2.5,
                                                                correction=_dev(corr, cuda))
        pair, weight, tiles, out = (t.cpu().numpy() for t in (pair, weight, tiles, out))
        n = int(n_tiles)
        assert n <= most
        owner = np.full(rows * top, -1)
        for g, r0, k, _ in tiles[:n]:
            assert 0 < k <= tile and (owner[r0:r0 + k] == -1).all()
            owner[r0:r0 + k] = g
        assert (owner >= 0).all() and sorted(pair.ravel().tolist()) == list(range(rows * top))
        close = 0
        for r in range(rows):
            chosen, s = kr.route(z[r].astype(float), corr.astype(float), top, groups, keep, 2.5)
            if owner[pair[r]].tolist() != chosen.tolist():   # only where two choice scores, or two groups, differ by rounding
                choice = np.sort(kr.sigmoid(z[r].astype(float)) + corr)
                close += 1
                assert np.diff(choice).min() < 1e-6
                continue
            assert np.abs(weight[r] - s).max() < 2e-6 * 2.5
            assert (out[pair[r]] == h[r]).all()
        assert close <= rows // 50


def test_route_variants(cuda):
    """Every combination of scores, group score, correction and weights."""
    rng = np.random.default_rng(2)
    rows, experts, top, groups, keep = 90, 24, 4, 6, 3
    z, h = 2 * _f32(rng, rows, experts), _f32(rng, rows, 8)
    for sigmoid in (False, True):
        for best in (1, 2):
            for corr in (None, rng.uniform(-0.2, 0.2, experts).astype(np.float32)):
                for scale in (0.0, 1.5):
                    pair, weight, tiles, n_tiles, _, _ = ops.moe_route(experts, top, groups, keep, 16, _dev(z, cuda), _dev(h, cuda), sigmoid=sigmoid, group_best=best, weight_scale=scale,
                                                                       correction=None if corr is None else _dev(corr, cuda))
                    owner = np.repeat(tiles[:int(n_tiles), 0].cpu().numpy(), tiles[:int(n_tiles), 2].cpu().numpy())
                    for r in range(rows):
                        s = kr.sigmoid(z[r].astype(float)) if sigmoid else np.exp(z[r].astype(float)) / np.exp(z[r].astype(float)).sum()
                        choice = s + (0 if corr is None else corr)
                        order = choice if sigmoid or corr is not None else z[r].astype(float)   # uncorrected softmax scores choose like their logits
                        gs = np.sort(order.reshape(groups, -1), axis=1)[:, -best:].sum(axis=1)
                        allowed = np.where(np.isin(np.arange(experts) // 4, np.argsort(-gs, kind="stable")[:keep]), choice, -np.inf)
                        chosen = np.argsort(-allowed, kind="stable")[:top]
                        w = s[chosen] / (s[chosen].sum() + 1e-20) * scale if scale else s[chosen]
                        assert owner[pair[r].cpu().numpy()].tolist() == chosen.tolist(), (sigmoid, best, scale)
                        assert np.abs(weight[r].cpu().numpy() - w).max() < 2e-6


@pytest.mark.parametrize("rows,experts,top,w,f", [(1, 4, 2, 40, 24), (9, 6, 3, 64, 13), (64, 16, 4, 136, 72), (300, 3, 2, 264, 136), (900, 7, 4, 320, 264)])
@pytest.mark.parametrize("tile", [8, 16, 32, 64, 128])
def test_grouped_matmuls_with_squared_relu(cuda, rows, experts, top, w, f, tile):
    rng = np.random.default_rng(rows + f)
    bf16 = tile != 8
    fp, wp = (f + 7) // 8 * 8, (w + 7) // 8 * 8
    up = kr.to_bf16((_f32(rng, experts, f, w) / w ** 0.5).astype(np.float32))
    down = kr.to_bf16((_f32(rng, experts, w, f) / f ** 0.5).astype(np.float32))
    h = np.zeros((rows, wp), np.float32)
    h[:, :w] = kr.to_bf16(_f32(rng, rows, w))
    z = _f32(rng, rows, experts)
    z[:, 0] += 1.0   # unequal shares
    dt = torch.bfloat16 if bf16 else torch.float32
    pair, _, tiles, n_tiles, srt, most = ops.moe_route(experts, top, 1, 1, tile, _dev(z, cuda), _dev(h, cuda, dt), sigmoid=True, group_best=2)
    gu, dn = np.zeros((experts, fp, wp), np.float32), np.zeros((experts, wp, fp), np.float32)
    gu[:, :f, :w], dn[:, :w, :f] = up, down
    status = torch.zeros(1, dtype=torch.int32, device=cuda)
    kw = dict(tiles=tiles, n_tiles=n_tiles, max_tiles=most, tile_rows=tile, batch=experts)
    if bf16:
        a = ops.dense_bf16(srt, _dev(gu, cuda, dt), rows * top, fp, wp, relu2=True, status=status, **kw)
        y = ops.dense_bf16(a, _dev(dn, cuda, dt), rows * top, wp, fp, out_f32=True, status=status, **kw)
    else:
        a = ops.dense_f32(srt, _dev(gu.transpose(0, 2, 1), cuda), rows * top, fp, wp, relu2=True, **kw)
        y = ops.dense_f32(a, _dev(dn.transpose(0, 2, 1), cuda), rows * top, wp, fp, **kw)
    assert int(status) == 0
    pair, a, y = pair.cpu().numpy(), a.float().cpu().numpy(), y.cpu().numpy()
    for r in range(0, rows, max(1, rows // 60)):
        for k, e in enumerate(np.argsort(-z[r].astype(float), kind="stable")[:top]):
            mid = kr.relu2(h[r, :w].astype(float) @ up[e].T)
            want = mid @ down[e].T
            assert np.abs(a[pair[r, k], :f] - mid).max() < (2 ** -7 * np.abs(mid).max() + 1e-3 if bf16 else 1e-5), (r, k)
            assert np.abs(y[pair[r, k], :w] - want).max() < (2e-2 if bf16 else 1e-5) * max(1.0, np.abs(want).max()), (r, k)


# ---- differential attention ----------------------------------------------------------------------------------------------
class _Cache:
    """Sequences of given lengths in scattered pages; projection rows on the device."""

    def __init__(self, rng, cuda, a, lens):
        self.a, self.cuda, self.bf16 = a, cuda, a.dtype == ops.BF16
        self.dt = torch.bfloat16 if self.bf16 else torch.float32
        pages = [(n + 15) // 16 for n in lens]
        total = sum(pages) + 3
        perm, table, o = rng.permutation(total), np.zeros((len(lens), max(pages) + 1), np.int32), 0
        for s, n in enumerate(pages):
            table[s, :n] = perm[o:o + n]
            o += n
        self.table = _dev(table, cuda)
        # rows that nobody has written are poison: a result that touches one is not a number
        self.pool = torch.full((total * a.page_bytes // (2 if self.bf16 else 4),), float("nan"), device=cuda, dtype=self.dt)
        self.slot = [s for s, n in enumerate(lens) for _ in range(n)]
        self.pos = [p for n in lens for p in range(n)]

    def pack(self, a, q, k=None, v=None, g=None):
        """[n][H][maps][dim], [n][G][maps][dim], [n][G][vdim], [n][H][vdim] -> projection rows of layout `a`."""
        row = np.full((q.shape[0], a.q_row), 3.0, np.float32)
        for x, off, st in ((q, 0, a.q_head_stride), (k, a.k_offset, a.k_head_stride)):
            if x is None:
                continue
            for h in range(x.shape[1]):
                for m in range(x.shape[2]):
                    at = off + h * st + m * a.map_stride
                    row[:, at:at + a.map_stride] = 0   # what the padded weights give
                    row[:, at:at + a.dim] = x[:, h, m]
        for x, off, st in ((v, a.v_offset, a.v_head_stride), (g, a.g_offset, a.g_head_stride)):
            if x is not None:
                for h in range(x.shape[1]):
                    row[:, off + h * st:off + h * st + a.vdim] = x[:, h]
        return _dev(row, self.cuda, self.dt)

    def append(self, rows):
        ops.grouped_append(self.a, rows, _i32(self.pos, self.cuda), _i32(self.slot, self.cuda), self.table, self.pool)

    def tiles(self, a, slot, pos):
        t = ops.grouped_tile_tokens(a)
        first, count, i, n = [], [], 0, len(slot)
        while i < n:
            e = i + 1
            while e < n and e - i < t and slot[e] == slot[i] and pos[e] == pos[e - 1] + 1:
                e += 1
            first.append(i), count.append(e - i)
            i = e
        return _i32(first, self.cuda), _i32(count, self.cuda)

    def attend(self, a, d, slot, pos, mode, splits):
        got, status = ops.grouped_attention(a, d, self.pool, self.table, _i32(slot, self.cuda), _i32([p + 1 for p in pos], self.cuda), max(pos) + 1,
                                            tiles=self.tiles(a, slot, pos) if mode == "tc" else None, splits=splits if mode == "tc" else 1)
        assert int(status) == 0
        g = got.float().cpu().numpy()
        assert (g[:, :, a.vdim:] == 0).all()
        return g[:, :, :a.vdim]


def _attend(a, q, k, v, g, pos):
    """Queries q [n][H][maps][dim] at `pos` over the keys and values of one sequence, gates g or None -> [n][H][vdim]."""
    group, maps = a.heads // a.kv_heads, q.shape[2]
    out = np.zeros((len(pos), a.heads, a.vdim))
    for n, i in enumerate(pos):
        lo = max(0, i - a.mask_size + 1) if a.mask == gm.MASK_WINDOW else 0
        for h in range(a.heads):
            o = []
            for m in range(maps):
                s = k[lo:i + 1, h // group, m] @ q[n, h, m] * a.scale
                p = np.exp(s - s.max())
                o.append((p / p.sum()) @ v[lo:i + 1, h // group])
            out[n, h] = o[0] if maps == 1 else kr.rms(o[0] - a.lambda_ * o[1], a.head_eps) * a.head_scale
    return out if g is None else out * kr.sigmoid(g)


SHAPES = [  # heads, kv heads, dim, vdim, window (0: none), gate
    (1, 1, 8, 8, 5, True), (6, 2, 24, 40, 9, True), (4, 4, 96, 72, 63, True), (16, 2, 64, 128, 64, True), (5, 1, 40, 20, 65, False), (8, 4, 64, 256, 200, True),
    (12, 3, 72, 136, 0, True), (130, 1, 8, 16, 31, True), (2, 1, 272, 320, 50, True), (7, 7, 13, 5, 17, False), (40, 8, 16, 48, 0, True), (4, 1, 128, 128, 100, True)]


def _random(rng, n, a, maps=2):
    q, k = (kr.to_bf16(_f32(rng, n, h, maps, a.dim)) for h in (a.heads, a.kv_heads))
    v, g = (kr.to_bf16(_f32(rng, n, h, a.vdim)) for h in (a.kv_heads, a.heads))
    return q, k, v, g


def _layout(shape, mode, maps=2, **kw):
    heads, kv, dim, vdim, window, gate = shape
    return ops.grouped_layout(heads, kv, dim, vdim, gm.MASK_WINDOW if window else gm.MASK_CAUSAL, window, 1.7 * dim ** -0.5, bf16=mode != "f32", maps=maps, gate=gate, lam=0.7,
                              head_scale=0.4, head_eps=1e-4, **kw)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("maps", [1, 2])
def test_attention_prompt(cuda, shape, mode, maps):
    a = _layout(shape, mode, maps)
    if mode == "tc" and ops.grouped_tile_tokens(a) == 0:
        assert shape[2] > 192 or shape[3] > 256
        pytest.skip("these sizes belong to the plain kernel")
    rng = np.random.default_rng(shape[2] + shape[4])
    lens = [150, 1, 37, 16]
    c = _Cache(rng, cuda, a, lens)
    q, k, v, g = _random(rng, sum(lens), a, maps)
    gate = g if a.gate else None
    d = c.pack(a, q, k, v, gate)
    c.append(d)
    want, o = [], 0
    for n in lens:
        s = slice(o, o + n)
        want.append(_attend(a, q[s].astype(float), k[s].astype(float), v[s].astype(float), None if gate is None else g[s].astype(float), range(n)))
        o += n
    want = np.concatenate(want)
    for splits in ((1, 2, 5) if mode == "tc" else (1,)):
        got = c.attend(a, d, c.slot, c.pos, mode, splits)
        assert np.abs(got - want).max() < (2e-5 if mode == "f32" else 2 ** -8 * np.abs(want).max() + 1e-3), splits


@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("window", [1, 15, 16, 17, 64, 100, 128, 1000, 0])
@pytest.mark.parametrize("as_prompt", [False, True])
@pytest.mark.parametrize("part", [0, 1])
def test_attention_sees_exactly_the_window(cuda, mode, window, as_prompt, part):
    """One stored key of one part points along that part of the query and outweighs all others: the difference has all of its value while
    the window lets it through and no trace of it otherwise; just inside and outside the edge, at page borders, past the first block."""
    heads, kv, dim, vdim, n = 6, 2, 40, 24, 450
    a = ops.grouped_layout(heads, kv, dim, vdim, gm.MASK_WINDOW if window else gm.MASK_CAUSAL, window, 1.0, bf16=mode != "f32", maps=2, gate=True, lam=0.9, head_scale=0.5, head_eps=1e-4)
    rng = np.random.default_rng(window)
    c = _Cache(rng, cuda, a, [n])
    q, k, v, g = _random(rng, n, a)
    c.append(c.pack(a, q, k, v, g))
    for far in (0, 1, 15, 16, 17, 47, 48, 63, 64, 128, 200, 207, 208):
        edge = far + window if window else n   # the first position that does not see it
        at = sorted({p for p in (far, edge - 2, edge - 1, edge, edge + 1) if far <= p < n} | (set() if window else {n - 1}))
        if as_prompt:   # one run that crosses the edge
            at = list(range(max(at[0], at[-1] - 30), at[-1] + 1))
        qf = 0.1 * _f32(rng, len(at), heads, 2, dim)
        for h in range(heads):
            key = k[far, h // 3, part]
            qf[:, h, part] = 20.0 * key / np.linalg.norm(key)
        qf = kr.to_bf16(qf.astype(np.float32))
        gf = kr.to_bf16(_f32(rng, len(at), heads, vdim))
        d = c.pack(a, qf, np.zeros((len(at), kv, 2, dim)), np.zeros((len(at), kv, vdim)), gf)
        want = _attend(a, qf.astype(float), k.astype(float), v.astype(float), gf.astype(float), at)
        for splits in ((1, 3) if mode == "tc" else (1,)):
            got = c.attend(a, d, [0] * len(at), at, mode, splits)
            assert np.abs(got - want).max() < (1e-4 if mode == "f32" else 2e-2 * np.abs(want).max()), (far, at, splits)
        raw = _attend(a, qf.astype(float), k.astype(float), v.astype(float), None, at)
        for i, p in enumerate(at):   # the spike is where it should be, so that the comparison above means something
            if p > far and (not window or window > 8) and p > 8:
                value = v[far, np.arange(heads) // 3].astype(float) * (1 if part == 0 else -1)
                cos = np.einsum("hv,hv->h", raw[i], value) / np.linalg.norm(raw[i], axis=1) / np.linalg.norm(value, axis=1)
                assert (cos.mean() > 0.6) == (p < edge), (far, p, cos)


@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
def test_attention_with_another_layers_keys(cuda, mode):
    """Rows of queries and gates only, more heads and another window over the same pages."""
    shape = (4, 2, 24, 40, 20, True)
    a, b = _layout(shape, mode), _layout((8, 2, 24, 40, 55, True), mode, shared_kv=True)
    assert b.page_bytes == a.page_bytes and b.q_row < a.q_row * 2
    rng = np.random.default_rng(4)
    n = 130
    c = _Cache(rng, cuda, a, [n])
    q, k, v, g = _random(rng, n, a)
    c.append(c.pack(a, q, k, v, g))
    q2, _, _, g2 = _random(rng, n, b)
    got = c.attend(b, c.pack(b, q2, g=g2), c.slot, c.pos, mode, 1)
    want = _attend(b, q2.astype(float), k.astype(float), v.astype(float), g2.astype(float), range(n))
    assert np.abs(got - want).max() < (2e-5 if mode == "f32" else 2 ** -8 * np.abs(want).max() + 1e-3)
    with pytest.raises(Exception, match="no keys"):
        ops.grouped_append(b, c.pack(b, q2, g=g2), _i32(c.pos, cuda), _i32(c.slot, cuda), c.table, c.pool)


def test_decode_equals_prompt_rows(cuda):
    """The same rows as one prompt, as single-token tiles with split keys, and mixed with another sequence's."""
    a = _layout((8, 2, 72, 40, 170, True), "tc")
    rng = np.random.default_rng(3)
    c = _Cache(rng, cuda, a, [300, 77])
    q, k, v, g = _random(rng, 377, a)
    d = c.pack(a, q, k, v, g)
    c.append(d)
    whole = c.attend(a, d, c.slot, c.pos, "tc", 1)
    for pick in ([5], [299, 376], [0, 300, 64, 169, 310, 170, 171, 299]):
        for splits in (1, 2, 3, 4, 9):
            got = c.attend(a, d[pick].contiguous(), [c.slot[i] for i in pick], [c.pos[i] for i in pick], "tc", splits)
            assert np.abs(got - whole[pick]).max() < 2 ** -7 * np.abs(whole).max()


# ---- latent attention with a query latent --------------------------------------------------------------------------------
@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("heads,dim,rot,rank,q_rank", [(3, 14, 6, 21, 5), (4, 16, 8, 64, 40), (2, 72, 70, 130, 200), (20, 8, 2, 8, 8)])
def test_latent_append_in_two_steps(cuda, bf16, heads, dim, rot, rank, q_rank):
    """Query latent, page and rotated queries against the equations; then the page through the attention over everything."""
    a = ops.latent_layout(heads, dim, rot, 16, rank, 0, 0.3 * (rank + rot) ** -0.5, bf16=bf16, q_rank=q_rank)
    rng = np.random.default_rng(rank)
    lens, dt = [70, 3], torch.bfloat16 if bf16 else torch.float32
    slot, pos = [0] * 70 + [1] * 3, list(range(70)) + list(range(3))
    n = len(pos)
    table = _dev(rng.permutation(10)[:10].reshape(2, 5).astype(np.int32), cuda)
    pool = torch.full((10 * a.page_bytes // (2 if bf16 else 4),), float("nan"), device=cuda, dtype=dt)
    rnd = kr.to_bf16 if bf16 else (lambda x: x)
    kv = np.zeros((n, a.kv_row), np.float32)
    raw_q, raw_l, raw_r = rnd(3 * _f32(rng, n, q_rank)), rnd(_f32(rng, n, rank)), rnd(_f32(rng, n, rot))
    kv[:, :q_rank], kv[:, a.dkv_offset:a.dkv_offset + rank], kv[:, a.rot_offset:a.rot_offset + rot] = raw_q, raw_l, raw_r
    nw, qw = rnd((1 + 0.3 * _f32(rng, rank)).astype(np.float32)), rnd((1 + 0.3 * _f32(rng, q_rank)).astype(np.float32))
    base = 50.0
    ang = np.arange(80)[:, None] * base ** (-np.arange(0, rot, 2) / rot)
    cos, sin = _dev(np.cos(ang).astype(np.float32), cuda), _dev(np.sin(ang).astype(np.float32), cuda)
    p, s = _i32(pos, cuda), _i32(slot, cuda)
    ql = ops.latent_append_keys(a, _dev(kv, cuda, dt), p, s, table, _dev(nw, cuda), _dev(qw, cuda), 1e-3, cos, sin, pool).float().cpu().numpy()
    want = kr.rms(raw_q.astype(float), 1e-3) * qw
    assert np.abs(ql[:, :q_rank] - want).max() < (2 ** -8 * np.abs(want).max() if bf16 else 1e-5) and (ql[:, q_rank:] == 0).all()
    # queries: the absorbed parts are the caller's, the rotated ones are written beside them
    absorbed, raw = rnd(_f32(rng, n, heads, rank)), rnd(_f32(rng, n, heads, dim + rot))
    q = np.zeros((n, heads, a.q_head_stride), np.float32)
    q[:, :, :dim], q[:, :, a.q_rot_offset:a.q_rot_offset + rot] = raw[:, :, :dim], raw[:, :, dim:]
    qa = np.zeros((n, heads, a.qa_head_stride), np.float32)
    qa[:, :, :rank] = absorbed
    d_qa = _dev(qa, cuda, dt)
    ops.latent_rotate_queries(a, _dev(q.reshape(n, -1), cuda, dt), p, cos, sin, d_qa)
    at = np.asarray(pos)
    q_rot, k_rot = kr.rotate(raw[:, :, dim:].astype(float), at, base), kr.rotate(raw_r.astype(float), at, base)
    got = d_qa.float().cpu().numpy()
    assert np.abs(got[:, :, a.qa_rot_offset:a.qa_rot_offset + rot] - q_rot).max() < (2 ** -8 * np.abs(q_rot).max() if bf16 else 1e-5)
    assert np.array_equal(got[:, :, :rank], absorbed)
    lat = kr.rms(raw_l.astype(float), 1e-3) * nw
    full_q = np.concatenate([absorbed, q_rot], -1)
    for mode in ("plain", "tc") if bf16 else ("plain",):
        t = max(ops.latent_tile_tokens(a), 1)
        first = [o + i for o, m in ((0, 70), (70, 3)) for i in range(0, m, t)]
        count = [min(t, (70 if f < 70 else 73) - f) for f in first]
        out, status = ops.latent_attention(a, d_qa, pool, table, s, _i32([x + 1 for x in pos], cuda), 70, tiles=(_i32(first, cuda), _i32(count, cuda)) if mode == "tc" else None)
        out = out.float().cpu().numpy()[:, :, :rank]
        assert int(status) == 0
        o = 0
        for m in lens:
            sl = slice(o, o + m)
            ref = kr.softmax_attention(full_q[sl], np.concatenate([lat, k_rot], 1)[sl][:, None], lat[sl][:, None], a.scale)
            assert np.abs(out[sl] - ref).max() < (1.2e-2 * np.abs(ref).max() if bf16 else 2e-5), mode
            o += m
