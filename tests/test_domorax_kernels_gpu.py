"""Domorax's mechanisms one by one, each through the C ABI against a plain reference of the same equation: the step with norms in groups and
an average over depth, the polynomial of normed powers, attention whose values are keys (convolutions with their state, norms, linear distance
bias, reach), latent attention with sinks, the delta rule with a decay per head and silu gates."""
import numpy as np
import pytest
import torch

from gptrs_b200 import model as gm
from gptrs_b200 import ops
from oracle import domorax_ref as dr

pytestmark = pytest.mark.gpu


def _dev(a, cuda, dt=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).to(cuda)
    return t if dt is None else t.to(dt)


def _i32(a, cuda):
    return torch.tensor(list(a), dtype=torch.int32, device=cuda)


def _f32(rng, *shape):
    return rng.standard_normal(shape).astype(np.float32)


# ---- the step between sublayers ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dim,groups", [(24, 1), (39, 3), (256, 2), (512, 4), (500, 5), (768, 6), (1024, 1), (2048, 8), (3072, 2), (3072, 3), (4096, 32), (6144, 3), (8192, 1), (9000, 9)])
def test_depth_step(cuda, dim, groups):
    rng = np.random.default_rng(dim + groups)
    n, states_n, eps, m = 13, 6, 1e-3, 0.37
    x, y = _f32(rng, n, dim), 3 * _f32(rng, n, dim) * np.repeat(10.0 ** rng.uniform(-1, 1, groups), dim // groups).astype(np.float32)
    g, gf = 1 + 0.3 * _f32(rng, dim), 1 + 0.3 * _f32(rng, dim)
    want = x + m * dr.group_rms(y.astype(float), groups, eps) * g
    kw = dict(y=_dev(y, cuda), gamma_out=_dev(g, cuda))
    gx, out = _dev(x, cuda), torch.empty(n, dim, device=cuda)
    h = ops.depth_step(groups, eps, m, gx, out, **kw)
    assert np.abs(out.cpu().numpy() - want).max() < 3e-5 and torch.equal(h, out) and np.array_equal(gx.cpu().numpy(), x)
    h = ops.depth_step(groups, eps, m, gx, gx, **kw, out_dtype=torch.bfloat16, ldh=dim + 8)   # in place; columns past the row are zeroed
    assert torch.equal(gx, out) and torch.equal(h[:, :dim], out.bfloat16()) and not h[:, dim:].any()
    # the end of a layer: any number of earlier results, the last one written
    for earlier in (1, 2, states_n - 1):
        a = _f32(rng, earlier + 1)
        st = _f32(rng, states_n, n, dim)
        st[earlier] = np.nan
        avg = np.einsum("j,jnd->nd", a[:-1].astype(float), st[:earlier].astype(float)) + a[-1] * want
        ds = _dev(st, cuda)
        h = ops.depth_step(groups, eps, m, _dev(x, cuda), out, **kw, states=ds, weights=_dev(a, cuda))
        assert np.abs(out.cpu().numpy() - avg).max() < 5e-5 and torch.equal(h, out)
        assert np.abs(ds[earlier].cpu().numpy() - want).max() < 3e-5 and np.array_equal(ds[:earlier].cpu().numpy(), st[:earlier])
        # the end of the model: listed rows, final norm, nothing written
        rows = [12, 0, 7]
        final = dr.group_rms(avg, groups, eps) * gf
        ds[earlier] = 5.0
        before, x2 = ds.clone(), _dev(x, cuda)
        h = ops.depth_step(groups, eps, m, x2, x2, **kw, states=ds, weights=_dev(a, cuda), gamma_in=_dev(gf, cuda), rows=_i32(rows, cuda))
        assert np.abs(h.cpu().numpy() - final[rows]).max() < 1e-4 and torch.equal(ds, before) and np.array_equal(x2.cpu().numpy(), x)
    h = ops.depth_step(groups, eps, x=_dev(want.astype(np.float32), cuda), gamma_in=_dev(gf, cuda))   # a norm alone
    assert np.abs(h.cpu().numpy() - dr.group_rms(want, groups, eps) * gf).max() < 1e-4


@pytest.mark.parametrize("dim,groups", [(39, 3), (256, 2), (1024, 2), (3072, 4)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_depth_step_sums_up_experts(cuda, dim, groups, dt):
    """The weighted sum of the experts' rows, plus a second output under a gate that lies in a column of a wider matrix."""
    rng = np.random.default_rng(dim)
    n, top, eps = 40, 3, 1e-5
    ld = (dim + 7) // 8 * 8
    ys, add, x = np.zeros((n * top, ld), np.float32), np.zeros((n, ld), np.float32), _f32(rng, n, dim)
    ys[:, :dim], add[:, :dim] = dr.to_bf16(_f32(rng, n * top, dim)), dr.to_bf16(_f32(rng, n, dim))
    pair, w, gate, g = rng.permutation(n * top).reshape(n, top).astype(np.int32), rng.uniform(0, 1, (n, top)).astype(np.float32), 3 * _f32(rng, n, 5), 1 + 0.3 * _f32(rng, dim)
    y = np.einsum("nk,nkd->nd", w.astype(float), ys[pair][:, :, :dim].astype(float))
    for gated in (None, gate):
        total = y + add[:, :dim] * (1 if gated is None else dr.sigmoid(gate[:, :1].astype(float)))
        want = x + 0.5 * dr.group_rms(total, groups, eps) * g
        h = ops.depth_step(groups, eps, 0.5, _dev(x, cuda), y=_dev(ys, cuda, dt), gamma_out=_dev(g, cuda), pair=_dev(pair, cuda), pair_weight=_dev(w, cuda), add=_dev(add, cuda, dt),
                           add_gate=None if gated is None else _dev(gate, cuda))
        assert np.abs(h.cpu().numpy() - want).max() < 3e-5


def test_depth_step_embedding(cuda):
    rng = np.random.default_rng(1)
    for dim, groups in ((40, 5), (256, 2)):
        e = _f32(rng, 30, dim)
        status, out = torch.zeros(1, dtype=torch.int32, device=cuda), torch.empty(6, dim, device=cuda)
        h = ops.depth_step(groups, 1e-5, embed=_dev(e, cuda), tokens=_i32([3, 29, 0, 3, 7, 1], cuda), x_out=out, status=status)
        assert np.array_equal(out.cpu().numpy(), e[[3, 29, 0, 3, 7, 1]]) and torch.equal(h, out) and int(status) == 0
        ops.depth_step(groups, 1e-5, embed=_dev(e, cuda), tokens=_i32([3, 30, 0, 3, 7, 1], cuda), x_out=out, status=status)
        assert int(status) == 2
    with pytest.raises(Exception, match="whole number"):
        ops.depth_step(7, 1e-5, x=torch.zeros(2, 40, device=cuda))


@pytest.mark.parametrize("n", [5, 48, 200, 512, 700, 1024, 2000, 3000, 6144, 9216, 16384, 20000])
@pytest.mark.parametrize("bf16", [False, True])
def test_poly_norm(cuda, n, bf16):
    rng = np.random.default_rng(n)
    rows, dt = 9, torch.bfloat16 if bf16 else torch.float32
    ld = (n + 7) // 8 * 8 if bf16 else n
    z = np.full((rows, ld), 7.0, np.float32)   # what lies past a row does not count
    z[:, :n] = dr.to_bf16(2 * _f32(rng, rows, n))
    z[3] *= 1e-2
    act = np.array([0.7, -0.4, 1.3, 0.2], np.float32)
    want = dr.poly_norm(z[:, :n].astype(float), act.astype(float), 1e-4)
    d = _dev(z, cuda, dt)
    y = ops.poly_norm(d, _dev(act, cuda), 1e-4, n)
    got = y.float().cpu().numpy()
    assert np.abs(got[:, :n] - want).max() < (2 ** -8 if bf16 else 3e-6) * max(1.0, np.abs(want).max()) and (got[:, n:] == 0).all()
    ops.poly_norm(d, _dev(act, cuda), 1e-4, n, out=d)
    assert torch.equal(d, y)


# ---- attention ---------------------------------------------------------------------------------------------------------
class _Cache:
    """Sequences in scattered pages, convolution states, and the same on the host: raw queries, keys and values go in, rows of any cut."""

    def __init__(self, rng, cuda, a, lens, gain_scale=1.0):
        self.a, self.cuda, self.bf16, self.lens = a, cuda, a.dtype == ops.BF16, lens
        self.dt = torch.bfloat16 if self.bf16 else torch.float32
        rnd = dr.to_bf16 if self.bf16 else (lambda x: x)
        pages = [(n + 15) // 16 for n in lens]
        perm, table, o = rng.permutation(sum(pages) + 3), np.zeros((len(lens), max(pages) + 1), np.int32), 0
        for s, n in enumerate(pages):
            table[s, :n] = perm[o:o + n]
            o += n
        self.table = _dev(table, cuda)
        # rows that nobody has written are poison: a result that touches one is not a number
        self.pool = torch.full(((sum(pages) + 3) * a.page_bytes // (2 if self.bf16 else 4),), float("nan"), device=cuda, dtype=self.dt)
        self.state = torch.full((len(lens), max(a.conv_floats, 1)), 9.0, device=cuda)   # what a slot's last user left must not show
        self.parity = [0] * len(lens)
        self.q, self.k = ([rnd(_f32(rng, n, h, a.dim)) for n in lens] for h in (a.heads, a.kv_heads))
        self.v = [rnd(_f32(rng, n, a.kv_heads, a.vdim)) for n in lens]
        self.qw, self.kw = (0.5 * _f32(rng, h, a.dim, max(a.taps, 1)) for h in (a.heads, a.kv_heads))
        for w in (self.qw, self.kw):
            w[..., -1] += 0.7
        self.gq, self.gk = gain_scale * (1 + 0.3 * _f32(rng, a.dim)), 1 + 0.3 * _f32(rng, a.dim)

    def mechanism(self, s):
        """Queries, keys and values [T][..][..] of a sequence as attention sees them."""
        a = self.a
        conv = lambda x, w: dr.short_conv(x.reshape(len(x), -1).astype(float), w.reshape(-1, w.shape[-1]).astype(float)).reshape(x.shape)  # noqa: E731
        q, k = (conv(self.q[s], self.qw), conv(self.k[s], self.kw)) if a.taps else (self.q[s].astype(float), self.k[s].astype(float))
        v = k if a.tied else self.v[s].astype(float)
        return (dr.rms(q, a.head_eps) * self.gq, dr.rms(k, a.head_eps) * self.gk, v) if a.qk_norm else (q, k, v)

    def prepare(self, parts):
        """parts: (slot, first position, rows); returns the queries, slots and positions of the rows."""
        a, cuda = self.a, self.cuda
        row = np.full((sum(n for _, _, n in parts), a.q_row), 3.0, np.float32)
        cols, o = [], 0
        for s, p, n in parts:
            for x, off, st, w in ((self.q, 0, a.q_head_stride, a.dim), (self.k, a.k_offset, a.k_head_stride, a.dim), (self.v, a.v_offset, a.v_head_stride, a.vdim)):
                if x is self.v and a.tied:
                    continue
                for h in range(x[s].shape[1]):
                    row[o:o + n, off + h * st:off + (h + 1) * st] = 0   # what the padded weights give
                    row[o:o + n, off + h * st:off + h * st + w] = x[s][p:p + n, h]
            cols += [(s, p + i, o, o + n - 1, self.parity[s]) for i in range(n)]
            o += n
            self.parity[s] ^= 1
        conv = np.zeros((max(a.taps, 1), a.conv_channels), np.float32)
        for w, off, st in ((self.qw, 0, a.q_head_stride), (self.kw, a.k_offset, a.k_head_stride)):
            for h in range(w.shape[0]):
                conv[:, off + h * st:off + h * st + a.dim] = w[h].T
        slot, pos, first, last, par = zip(*cols)
        q = ops.grouped_prepare(a, _dev(row, cuda, self.dt), _dev(conv, cuda) if a.taps else None, _dev(self.gq * self.gk if a.tied else self.gq, cuda), _dev(self.gk, cuda), self.state,
                                tuple(_i32(c, cuda) for c in (slot, pos, first, last, par)), self.table, self.pool)
        return q, list(slot), list(pos)

    def tiles(self, slot, pos):
        t = ops.grouped_tile_tokens(self.a)
        first, count, i, n = [], [], 0, len(slot)
        while i < n:
            e = i + 1
            while e < n and e - i < t and slot[e] == slot[i] and pos[e] == pos[e - 1] + 1:
                e += 1
            first.append(i), count.append(e - i)
            i = e
        return _i32(first, self.cuda), _i32(count, self.cuda)

    def attend(self, q, slot, pos, r1, mode, splits, reach=None):
        got, status = ops.grouped_attention(self.a, q, self.pool, self.table, _i32(slot, self.cuda), _i32([p + 1 for p in pos], self.cuda), max(pos) + 1,
                                            None if r1 is None else _dev(np.asarray(r1, np.float32), self.cuda), reach=None if reach is None else _i32(reach, self.cuda),
                                            tiles=self.tiles(slot, pos) if mode == "tc" else None, splits=splits if mode == "tc" else 1)
        assert int(status) == 0
        g = got.float().cpu().numpy()
        assert (g[:, :, self.a.vdim:] == 0).all()
        return g[:, :, :self.a.vdim]


def _attend(a, q, k, v, pos, r1):
    """Queries q [n][H][dim] at `pos` over keys and values of one sequence -> [n][H][vdim]."""
    group = a.heads // a.kv_heads
    out = np.zeros((len(pos), a.heads, a.vdim))
    for n, i in enumerate(pos):
        lo = max(0, i - a.mask_size + 1) if a.mask == gm.MASK_WINDOW else 0
        for h in range(a.heads):
            s = k[lo:i + 1, h // group] @ q[n, h] * a.scale
            if a.softcap:
                s = a.softcap * np.tanh(s / a.softcap)
            out[n, h] = dr.softmax_sink(s - (0 if r1 is None else r1[h]) * (i - np.arange(lo, i + 1))) @ v[lo:i + 1, h // group]
    return out


SHAPES = [  # heads, kv heads, dim, vdim (None: tied), taps, norms, linear bias, window, soft cap
    (1, 1, 8, None, 1, 1, 1, 0, 0), (6, 2, 24, None, 3, 1, 1, 0, 0), (8, 2, 96, None, 4, 1, 1, 0, 0), (16, 2, 128, None, 2, 1, 1, 0, 0), (5, 1, 13, None, 4, 1, 1, 0, 0),
    (32, 4, 64, None, 4, 1, 1, 0, 0), (130, 1, 16, None, 4, 1, 1, 0, 0), (4, 2, 192, None, 5, 1, 1, 0, 0), (2, 2, 256, None, 3, 1, 1, 0, 0), (2, 1, 272, None, 4, 1, 1, 0, 0),
    (4, 4, 40, None, 0, 1, 1, 33, 0), (6, 3, 20, None, 4, 0, 0, 0, 0), (8, 2, 72, 40, 4, 1, 1, 0, 0), (4, 1, 24, 72, 7, 1, 1, 70, 0), (3, 3, 64, 128, 2, 0, 1, 0, 9.0), (8, 4, 32, 16, 0, 1, 0, 0, 0),
    (7, 7, 7, None, 9, 1, 1, 0, 12.0), (4, 2, 24, 24, 0, 0, 1, 0, 0)]


def _layout(shape, mode):
    heads, kv, dim, vdim, taps, norm, bias, window, cap = shape
    return ops.grouped_layout(heads, kv, dim, dim if vdim is None else vdim, gm.MASK_WINDOW if window else gm.MASK_CAUSAL, window, 1.7 * dim ** -0.5, cap,
                              gm.DISTANCE_LINEAR if bias else gm.DISTANCE_NONE, bf16=mode != "f32", head_eps=1e-4, taps=taps, qk_norm=norm, tied=vdim is None)


def _slopes(a):
    return np.array([dr.slope(h, a.heads) for h in range(a.heads)]) if a.distance_bias else None


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
def test_attention_over_any_cut(cuda, shape, mode):
    """Convolutions that carry their state over portions down to one token, with slots that held something else before; every row against the
    whole sequence."""
    a = _layout(shape, mode)
    if mode == "tc" and ops.grouped_tile_tokens(a) == 0:
        assert shape[2] > 256
        pytest.skip("these sizes belong to the plain kernel")
    rng = np.random.default_rng(shape[2] + shape[4])
    lens = [150, 1, 37, 16]
    c = _Cache(rng, cuda, a, lens)
    if a.taps == 0 and not a.qk_norm and not a.tied:   # nothing to prepare: the projection rows are appended
        with pytest.raises(Exception, match="append"):
            c.prepare([(0, 0, 5)])
        return
    r1 = _slopes(a)
    want = [_attend(a, *c.mechanism(s), range(n), r1) for s, n in enumerate(lens)]
    top = max(np.abs(w).max() for w in want)
    for cuts in ([1000], [1], [2, 1, 3, 19, 1, 1, 40], [16, 17, 1, 64]):
        at, i = [0] * len(lens), 0
        c.parity = [int(x) for x in rng.integers(0, 2, len(lens))]
        while any(p < n for p, n in zip(at, lens)):
            parts = []
            for s in rng.permutation(len(lens)):
                m = min(cuts[i % len(cuts)], lens[s] - at[s])
                i += 1
                if m > 0 and (len(cuts) == 1 or rng.random() < 0.8):
                    parts.append((int(s), at[s], m))
            if not parts:
                continue
            q, slot, pos = c.prepare(parts)
            ref = np.concatenate([want[s][p:p + m] for s, p, m in parts])
            for splits in ((1, 3) if mode == "tc" else (1,)):
                got = c.attend(q, slot, pos, r1, mode, splits)
                assert np.abs(got - ref).max() < (5e-5 * max(1.0, top) if mode == "f32" else 1.5e-2 * top), (cuts, parts, splits)
            for s, _, m in parts:
                at[s] += m


def test_prepare_of_many_rows(cuda):
    """More rows than the one-row-per-warp form takes: runs that start and end inside a warp's rows, a run shorter than the state among them."""
    for shape in ((6, 2, 24, None, 4, 1, 1, 0, 0), (4, 2, 200, None, 3, 1, 1, 0, 0), (4, 2, 24, 40, 2, 1, 1, 0, 0)):
        a = _layout(shape, "bf16")
        lens = [300, 1, 2, 37, 5]
        c = _Cache(np.random.default_rng(5), cuda, a, lens)
        ref = [c.mechanism(s) for s in range(len(lens))]
        at = [0] * len(lens)
        for parts in ([(3, 0, 30), (1, 0, 1), (0, 0, 270), (2, 0, 1), (4, 0, 2)], [(4, 2, 3), (0, 270, 30), (3, 30, 7), (2, 1, 1)]):
            q, _, _ = c.prepare(parts)
            got, o = q.float().cpu().numpy().reshape(len(q), a.heads, a.q_head_stride)[:, :, :a.dim], 0
            for s, p, n in parts:
                assert p == at[s]
                want = ref[s][0][p:p + n] * (c.gk if a.tied else 1)
                assert np.abs(got[o:o + n] - want).max() < 2 ** -8 * np.abs(want).max() + 1e-5, (s, p)
                o += n
                at[s] += n
        out = c.attend(q, [p[0] for p in parts for _ in range(p[2])], [p[1] + i for p in parts for i in range(p[2])], _slopes(a), "tc", 1)
        o = 0
        for s, p, n in parts:   # the pages
            want = _attend(a, ref[s][0][p:p + n], ref[s][1], ref[s][2], range(p, p + n), _slopes(a))
            assert np.abs(out[o:o + n] - want).max() < 1.5e-2 * np.abs(want).max()
            o += n


@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("as_prompt", [False, True])
@pytest.mark.parametrize("slope", [0.0, 0.02, 0.5])
def test_attention_finds_far_keys(cuda, mode, as_prompt, slope):
    """One stored key points along the query and outweighs all others, however far away, unless the distance costs more than it brings; at
    page and block borders, with split keys, and for positions of all kinds."""
    heads, kv, dim, n = 6, 2, 40, 450
    a = ops.grouped_layout(heads, kv, dim, dim, gm.MASK_CAUSAL, 0, 1.0, 0.0, gm.DISTANCE_LINEAR, bf16=mode != "f32", head_eps=1e-4, taps=3, qk_norm=True, tied=True)
    c = _Cache(np.random.default_rng(7), cuda, a, [n])
    _, _, _ = c.prepare([(0, 0, n)])
    _, k, v = c.mechanism(0)
    r1 = np.full(heads, slope)
    for far in (0, 1, 15, 16, 17, 47, 48, 63, 64, 128, 200, 207, 208, 385):
        at = sorted({p for p in (far, far + 1, far + 15, far + 16, far + 64, far + 100, n - 1) if p < n})
        if as_prompt:
            at = list(range(at[-2], min(at[-2] + 40, n)))
        qf = np.zeros((len(at), heads, dim), np.float32)
        for h in range(heads):
            key = k[far, h // 3]
            qf[:, h] = 20.0 * key / np.linalg.norm(key)
        row = np.zeros((len(at), a.query_row), np.float32)
        for h in range(heads):
            row[:, h * a.q_head_stride:h * a.q_head_stride + dim] = qf[:, h] * c.gk   # the keys' gain lies in the queries
        q = _dev(row, cuda, c.dt)
        stored = q.float().cpu().numpy().reshape(len(at), heads, -1)[:, :, :dim] / c.gk
        want = _attend(a, stored.astype(float), k, v, at, r1)
        for splits in ((1, 3, 7) if mode == "tc" else (1,)):
            got = c.attend(q, [0] * len(at), at, r1, mode, splits)
            assert np.abs(got - want).max() < (2e-4 if mode == "f32" else 3e-2 * np.abs(want).max()), (far, at, splits)
        if slope < 0.1:   # the spike is where it should be, so that the comparison above means something
            for i in range(len(at)):
                assert max(np.abs(want[i, h] - v[far, h // 3]).max() for h in range(heads)) < 0.3, (far, at[i])


@pytest.mark.parametrize("mode", ["f32", "tc"])
def test_reach_leaves_out_what_weighs_nothing(cuda, mode):
    """Norms bound the scores: what a steep head cannot see may be left out, and only that. Keys right at the reach are still there."""
    a = ops.grouped_layout(4, 2, 24, 24, gm.MASK_CAUSAL, 0, 0.1, 0.0, gm.DISTANCE_LINEAR, bf16=mode != "f32", head_eps=1e-4, taps=2, qk_norm=True, tied=True)
    n = 700
    c = _Cache(np.random.default_rng(8), cuda, a, [n])
    q, slot, pos = c.prepare([(0, 0, n)])
    r1 = [0.5, 0.4, 0.2, 0.1]
    bound = 0.1 * 24 * np.abs(c.gq * c.gk).max()
    reach = [int(np.ceil((2 * bound + 32) / r1[1])), int(np.ceil((2 * bound + 32) / r1[3]))]
    assert reach[0] < 200
    full, near = c.attend(q, slot, pos, r1, mode, 1), c.attend(q, slot, pos, r1, mode, 1, reach)
    assert np.abs(full - near).max() < (1e-6 if mode == "f32" else 2 ** -8 * np.abs(full).max())
    at = [0, 15, 16, 100, reach[0] + 1, 333, n - 1]
    got = c.attend(q[at].contiguous(), [0] * len(at), at, r1, mode, 3, reach)
    assert np.abs(got - full[at]).max() < (1e-6 if mode == "f32" else 2 ** -7 * np.abs(full).max())
    # without a bias the keys at the reach count as much as any: exactly those from there on are read
    flat = c.attend(q[[n - 1]].contiguous(), [0], [n - 1], [0.0] * 4, mode, 1, [64, 64])
    qm, km, vm = c.mechanism(0)
    lo = n - 1 - 64
    want = _attend(a, qm[n - 1:], km[lo:], vm[lo:], [n - 1 - lo], None)
    assert np.abs(flat - want).max() < (5e-5 if mode == "f32" else 1.5e-2 * np.abs(want).max())


def test_decode_equals_prompt_rows(cuda):
    """The same rows as one prompt, as single-token tiles with split keys, and mixed with another sequence's."""
    a = _layout((8, 2, 96, None, 4, 1, 1, 0, 0), "tc")
    c = _Cache(np.random.default_rng(3), cuda, a, [300, 77])
    q, slot, pos = c.prepare([(0, 0, 300), (1, 0, 77)])
    r1 = _slopes(a)
    whole = c.attend(q, slot, pos, r1, "tc", 1)
    for pick in ([5], [299, 376], [0, 300, 64, 169, 310, 170, 171, 299]):
        for splits in (1, 2, 3, 4, 9, 40):
            got = c.attend(q[pick].contiguous(), [slot[i] for i in pick], [pos[i] for i in pick], r1, "tc", splits)
            assert np.abs(got - whole[pick]).max() < 2 ** -7 * np.abs(whole).max()


# ---- latent attention with sinks -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("heads,rank,rot,window", [(3, 21, 6, 9), (8, 96, 32, 96), (20, 136, 72, 64), (70, 64, 8, 100), (130, 24, 8, 33), (4, 256, 64, 0)])
def test_latent_attention_with_sinks(cuda, mode, heads, rank, rot, window):
    """Sinks from nothing to all of the softmax, below and far above the scores; prompts and decode rows, with split keys."""
    a = ops.latent_layout(heads, 16, rot, 16, rank, window, 1.5 * (rank + rot) ** -0.5, bf16=mode != "f32", q_rank=8)
    rng = np.random.default_rng(rank + heads)
    dt, n = torch.bfloat16 if mode != "f32" else torch.float32, 210
    rnd = dr.to_bf16 if mode != "f32" else (lambda x: x)
    table = _dev(rng.permutation(14).reshape(1, 14).astype(np.int32), cuda)
    pool = torch.full((14 * a.page_bytes // (2 if mode != "f32" else 4),), float("nan"), device=cuda, dtype=dt)
    kv = np.zeros((n, a.kv_row), np.float32)
    raw = rnd(_f32(rng, n, rank + rot))
    kv[:, a.dkv_offset:a.dkv_offset + rank], kv[:, a.rot_offset:a.rot_offset + rot] = raw[:, :rank], raw[:, rank:]
    one = torch.ones(rank, device=cuda)
    zeros, still = torch.zeros(n, max(rot // 2, 1), device=cuda), torch.ones(n, max(rot // 2, 1), device=cuda)   # no rotation
    p, s = _i32(range(n), cuda), _i32([0] * n, cuda)
    ops.latent_append_keys(a, _dev(kv, cuda, dt), p, s, table, one, torch.ones(8, device=cuda), 1e-4, still, zeros, pool)
    key = np.concatenate([dr.rms(raw[:, :rank].astype(float), 1e-4), raw[:, rank:]], 1)
    q = rnd(_f32(rng, n, heads, rank + rot))
    qa = np.zeros((n, heads, a.qa_head_stride), np.float32)
    qa[:, :, :rank], qa[:, :, a.qa_rot_offset:a.qa_rot_offset + rot] = q[:, :, :rank], q[:, :, rank:]
    d_qa = _dev(qa, cuda, dt)
    sink = np.linspace(-3, 9, heads).astype(np.float32)
    sink[-1], sink[0] = 300.0, -300.0   # takes everything; takes nothing
    want = np.zeros((n, heads, rank))
    for i in range(n):
        lo = max(0, i - window + 1) if window else 0
        for h in range(heads):
            want[i, h] = dr.softmax_sink(key[lo:i + 1] @ q[i, h] * a.scale, sink[h].astype(float)) @ key[lo:i + 1, :rank]
    tol = 2e-5 if mode == "f32" else 1.2e-2 * np.abs(want).max()
    t = max(ops.latent_tile_tokens(a), 1)
    first = list(range(0, n, t))
    tiles = (_i32(first, cuda), _i32([min(t, n - f) for f in first], cuda))
    for splits in ((1, 2, 4) if mode == "tc" else (1,)):
        got, status = ops.latent_attention(a, d_qa, pool, table, s, _i32(range(1, n + 1), cuda), n, tiles=tiles if mode == "tc" else None, splits=splits, sink=_dev(sink, cuda))
        got = got.float().cpu().numpy()[:, :, :rank]
        assert int(status) == 0 and np.abs(got - want).max() < tol, splits
        assert not got[:, -1].any()
        at = [0, 1, 16, 63, 64, 150, n - 1]
        one_each = (_i32(range(len(at)), cuda), _i32([1] * len(at), cuda))
        got, status = ops.latent_attention(a, d_qa[at].contiguous(), pool, table, _i32([0] * len(at), cuda), _i32([x + 1 for x in at], cuda), n,
                                           tiles=one_each if mode == "tc" else None, splits=splits, sink=_dev(sink, cuda))
        assert int(status) == 0 and np.abs(got.float().cpu().numpy()[:, :, :rank] - want[at]).max() < tol, splits


# ---- delta rule with a decay per head --------------------------------------------------------------------------------------
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(1, 1, 8, 8, 4), (4, 2, 16, 24, 3), (6, 6, 32, 64, 4), (3, 1, 5, 7, 2), (2, 2, 64, 40, 1), (4, 4, 128, 128, 4), (2, 1, 100, 130, 5),
                                                    (2, 2, 200, 260, 4), (1, 1, 300, 33, 7), (12, 3, 32, 20, 4),
                                                    (16, 8, 72, 24, 4), (30, 10, 72, 24, 4)])   # columns per warp depend on the number of heads and runs
@pytest.mark.parametrize("bf16", [False, True])
def test_delta_rule_with_head_decays_over_any_cut(cuda, heads, kv, dim, vdim, taps, bf16):
    rng = np.random.default_rng(dim + vdim)
    a = ops.delta_layout(heads, kv, dim, vdim, taps, 0, 0, 1e-5, bf16=bf16, gate_silu=True)
    n, dt = 70, torch.bfloat16 if bf16 else torch.float32
    rnd = lambda x: dr.to_bf16(x.astype(np.float32)) if bf16 else x.astype(np.float32)  # noqa: E731
    ch = 2 * kv * dim + heads * vdim
    conv = (0.5 * rng.standard_normal((ch, taps))).astype(np.float32)
    a_log, dt_bias = np.log(rng.uniform(0.3, 3.0, heads)).astype(np.float32), rng.uniform(-6, 0, heads).astype(np.float32)
    norm = (1 + 0.3 * rng.standard_normal(vdim)).astype(np.float32)
    raw, beta, dec, gate = (rng.standard_normal((3, n, w)) for w in (ch, heads, heads, heads * vdim))
    raw[:, 40, :2 * kv * dim] *= 8.0     # keys that stand out
    raw, beta, dec, gate = (rnd(x) for x in (raw, beta, dec, gate))
    of = np.arange(heads) // (heads // kv)
    want = []
    for s in range(3):
        x = dr.silu(dr.short_conv(raw[s].astype(float), conv.astype(float)))
        q = (dr.unit(x[:, :kv * dim].reshape(n, kv, dim)) * dim ** -0.5)[:, of]
        k = dr.unit(x[:, kv * dim:2 * kv * dim].reshape(n, kv, dim))[:, of]
        g = np.repeat(dr.head_decay(dec[s].astype(float), a_log.astype(float), dt_bias.astype(float))[:, :, None], dim, 2)
        o = dr.delta_rule(q, k, x[:, 2 * kv * dim:].reshape(n, heads, vdim), g, dr.sigmoid(beta[s].astype(float)))
        want.append(dr.rms(o, 1e-5) * norm * dr.silu(gate[s].astype(float).reshape(n, heads, vdim)))

    def proj(s, lo, hi):
        row = np.full((hi - lo, a.row), 7.0, np.float32)
        for off, x in ((a.q_offset, raw[s, lo:hi, :kv * dim]), (a.k_offset, raw[s, lo:hi, kv * dim:2 * kv * dim]), (a.v_offset, raw[s, lo:hi, 2 * kv * dim:]),
                       (a.beta_offset, beta[s, lo:hi]), (a.a_offset, dec[s, lo:hi]), (a.g_offset, gate[s, lo:hi])):
            row[:, off:off + x.shape[1]] = x
        return row

    state = torch.full((3, a.state_floats), 9.0, device=cuda)            # what a slot's last user left must not show
    conv_state = torch.full((3, max(a.conv_floats, 1)), 9.0, device=cuda)
    consts = [_dev(x, cuda) for x in (conv, a_log, dt_bias, norm)]
    for cuts in ([n], [1], [2, 1, 3, 19, 1, 1, 40], [16, 17, 1, 36]):
        parity, at, i = [0, 1, 0], [0, 0, 0], 0
        while min(at) < n:
            parts = []
            for s in rng.permutation(3):
                m = min(cuts[i % len(cuts)], n - at[s])
                i += 1
                if m > 0 and rng.random() < 0.8:
                    parts.append((int(s), at[s], m))
            if not parts:
                continue
            cols, starts = [], []
            for s, p, m in parts:
                starts.append(len(cols))
                cols += [(s, p + j, starts[-1], starts[-1] + m - 1, parity[s]) for j in range(m)]
            got = ops.delta_rule(a, _dev(np.concatenate([proj(s, p, p + m) for s, p, m in parts]), cuda, dt), None, None, *consts, state, conv_state,
                                 tuple(_i32(c, cuda) for c in zip(*cols)), _i32(starts, cuda))
            w = np.concatenate([want[s][p:p + m] for s, p, m in parts])
            g = got.float().cpu().numpy()
            tol = 2 ** -8 * np.abs(w).max() + 1e-4 if bf16 else 5e-5 * max(1.0, np.abs(w).max())
            assert np.abs(g[:, :, :vdim] - w).max() < tol, (cuts, parts)
            assert (g[:, :, vdim:] == 0).all()
            for s, p, m in parts:
                at[s] += m
                parity[s] ^= 1
