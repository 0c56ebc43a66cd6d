"""Felepel's mechanisms one by one, each through the C ABI against a plain reference of the same equation: norms on both sides of a
sublayer, grouped matmuls, routing, attention with grouped heads (masks, soft cap, distance penalty, far keys, key splits), the delta
rule with its states over any cut."""
import numpy as np
import pytest
import torch

from gptrs_b200 import model as gm
from gptrs_b200 import ops
from oracle import felepel_ref as fr

pytestmark = pytest.mark.gpu


def _dev(a, cuda, dt=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).to(cuda)
    return t if dt is None else t.to(dt)


def _i32(a, cuda):
    return torch.tensor(list(a), dtype=torch.int32, device=cuda)


# ---- norms on both sides -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dim", [24, 37, 512, 700, 1028, 2048, 3072, 4100, 5001])
def test_norm_step(cuda, dim):
    rng = np.random.default_rng(dim)
    n = 19
    x, y = rng.standard_normal((n, dim)).astype(np.float32), 3 * rng.standard_normal((n, dim)).astype(np.float32)
    g, f = (1 + 0.3 * rng.standard_normal((2, dim))).astype(np.float32)
    want_x = x + fr.rms(y.astype(float), 1e-4) * g
    want_h = fr.rms(want_x, 1e-4) * f
    gx = _dev(x, cuda)
    h = ops.norm_step(gx, 1e-4, y=_dev(y, cuda), gamma_out=_dev(g, cuda), gamma_in=_dev(f, cuda))
    assert np.abs(gx.cpu().numpy() - want_x).max() < 1e-5 and np.abs(h.cpu().numpy() - want_h).max() < 2e-5
    gx = _dev(x, cuda)
    assert ops.norm_step(gx, 1e-4, y=_dev(y, cuda), gamma_out=_dev(g, cuda)) is None   # nothing follows
    assert np.abs(gx.cpu().numpy() - want_x).max() < 1e-5
    # bf16 in and out, padding columns, gathered rows: x is left alone
    yb, ldh = fr.to_bf16(y), (dim + 7) // 8 * 8
    rows = [18, 0, 0, 7]
    gx = _dev(x, cuda)
    h = ops.norm_step(gx, 1e-4, y=_dev(yb, cuda, torch.bfloat16), gamma_out=_dev(g, cuda), gamma_in=_dev(f, cuda), rows=_i32(rows, cuda), out_dtype=torch.bfloat16, ldh=ldh)
    want = (fr.rms(x + fr.rms(yb.astype(float), 1e-4) * g, 1e-4) * f)[rows]
    assert np.abs(h[:, :dim].float().cpu().numpy() - want).max() < 2 ** -8 * np.abs(want).max() and (h[:, dim:] == 0).all()
    assert np.array_equal(gx.cpu().numpy(), x)
    h = ops.norm_step(gx, 1e-4, gamma_in=_dev(f, cuda), rows=_i32(rows, cuda))   # no sublayer output
    assert np.abs(h.cpu().numpy() - (fr.rms(x.astype(float), 1e-4) * f)[rows]).max() < 2e-5


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_norm_step_sums_the_experts(cuda, dt):
    rng = np.random.default_rng(0)
    n, dim, top = 11, 72, 3
    x, y = rng.standard_normal((n, dim)).astype(np.float32), fr.to_bf16(rng.standard_normal((n * top, dim)).astype(np.float32))
    g, f = (1 + 0.3 * rng.standard_normal((2, dim))).astype(np.float32)
    pair, w = rng.permutation(n * top).reshape(n, top), rng.random((n, top)).astype(np.float32)
    want = x + fr.rms(np.einsum("nk,nkd->nd", w.astype(float), y[pair].astype(float)), 1e-5) * g
    gx = _dev(x, cuda)
    h = ops.norm_step(gx, 1e-5, y=_dev(y, cuda, dt), gamma_out=_dev(g, cuda), gamma_in=_dev(f, cuda), pair=_dev(pair.astype(np.int32), cuda), pair_weight=_dev(w, cuda))
    assert np.abs(gx.cpu().numpy() - want).max() < 1e-5 and np.abs(h.cpu().numpy() - fr.rms(want, 1e-5) * f).max() < 2e-5


def test_norm_step_embedding(cuda):
    rng = np.random.default_rng(1)
    v, d, n = 30, 44, 25
    table, pos_table, f = rng.standard_normal((v, d)).astype(np.float32), rng.standard_normal((n, d)).astype(np.float32), rng.standard_normal(d).astype(np.float32)
    tok, pos = rng.integers(0, v, n), rng.permutation(n)
    x = torch.zeros(n, d, device=cuda)
    kw = dict(embed=_dev(table, cuda), pos_embed=_dev(pos_table, cuda), gamma_in=_dev(f, cuda))
    h = ops.norm_step(x, 1e-6, tokens=_i32(tok, cuda), positions=_i32(pos, cuda), **kw)
    want = table[tok] + pos_table[pos]
    assert np.abs(x.cpu().numpy() - want).max() < 1e-6 and np.abs(h.cpu().numpy() - fr.rms(want.astype(float), 1e-6) * f).max() < 2e-5
    for t, p in ((v, 0), (-1, 0), (0, n), (0, -1)):   # out of range: flagged, nothing read outside the tables
        status = torch.zeros(1, dtype=torch.int32, device=cuda)
        tok2, pos2 = tok.copy(), pos.copy()
        tok2[4], pos2[4] = t, p
        ops.norm_step(x, 1e-6, tokens=_i32(tok2, cuda), positions=_i32(pos2, cuda), status=status, **kw)
        assert int(status) == 2


# ---- experts -----------------------------------------------------------------------------------------------------------
def _interleave(gate, up):
    """[E][F][W] each -> [E][2 F'][W], 8 gates, then their 8 partners; F' = F rounded up to 8."""
    e, f, w = gate.shape
    fp = (f + 7) // 8 * 8
    out = np.zeros((e, fp // 8, 2, 8, w), np.float32)
    for part, a in enumerate((gate, up)):
        padded = np.zeros((e, fp, w), np.float32)
        padded[:, :f] = a
        out[:, :, part] = padded.reshape(e, fp // 8, 8, w)
    return out.reshape(e, 2 * fp, w)


@pytest.mark.parametrize("rows,experts,top,groups,keep", [(1, 4, 2, 1, 1), (5, 12, 3, 4, 2), (64, 64, 4, 8, 3), (128, 33, 5, 3, 3), (129, 6, 6, 2, 2), (300, 1, 1, 1, 1),
                                                          (700, 96, 2, 6, 1), (1500, 512, 8, 16, 4), (37, 1024, 16, 1, 1)])
def test_route(cuda, rows, experts, top, groups, keep):
    rng = np.random.default_rng(rows + experts)
    z = (4 * rng.standard_normal((rows, experts))).astype(np.float32)
    h = rng.standard_normal((rows, 20)).astype(np.float32)
    for tile in (8, 16, 128):
        pair, weight, tiles, n_tiles, out, most = ops.moe_route(experts, top, groups, keep, tile, _dev(z, cuda), _dev(h, cuda))
        pair, weight, tiles, out = (t.cpu().numpy() for t in (pair, weight, tiles, out))
        n = int(n_tiles)
        assert n <= most
        owner = np.full(rows * top, -1)     # expert of every sorted row, from the tiles
        for g, r0, k, _ in tiles[:n]:
            assert 0 < k <= tile and (owner[r0:r0 + k] == -1).all()
            owner[r0:r0 + k] = g
        assert (owner >= 0).all() and (np.diff(owner) >= 0).all()
        assert sorted(pair.ravel().tolist()) == list(range(rows * top))
        for r in range(rows):
            chosen, s = fr.route(z[r].astype(float), top, groups, keep)
            assert owner[pair[r]].tolist() == chosen.tolist()
            assert np.abs(weight[r] - s).max() < 1e-6
            assert (out[pair[r]] == h[r]).all()


def test_route_again_with_the_same_counters(cuda):
    rng = np.random.default_rng(4)
    work = torch.zeros(4096, dtype=torch.int32, device=cuda)
    for rows, experts in ((400, 8), (3, 5), (130, 12), (400, 3), (400, 8)):   # as layers with unequal routers share them
        z = rng.standard_normal((rows, experts)).astype(np.float32)
        pair, _, tiles, n, _, _ = ops.moe_route(experts, 2, 1, 1, 16, _dev(z, cuda), torch.zeros(rows, 8, device=cuda), work=work)
        assert sorted(pair.flatten().tolist()) == list(range(2 * rows))
        assert int(tiles[:int(n), 2].sum()) == 2 * rows


@pytest.mark.parametrize("rows,experts,top,w,f", [(1, 4, 2, 40, 24), (9, 6, 3, 64, 13), (64, 16, 4, 136, 72), (100, 5, 2, 72, 200), (300, 3, 2, 264, 136), (900, 7, 4, 320, 264), (2000, 4, 2, 256, 512)])
@pytest.mark.parametrize("tile", [8, 16, 32, 64, 128])
def test_grouped_matmuls(cuda, rows, experts, top, w, f, tile):
    """silu(gate) up and down of every chosen expert, against the same rows computed expert by expert."""
    rng = np.random.default_rng(rows + f)
    bf16 = tile != 8
    fp, wp = (f + 7) // 8 * 8, (w + 7) // 8 * 8
    gate, up = (fr.to_bf16((rng.standard_normal((experts, f, w)) / w ** 0.5).astype(np.float32)) for _ in range(2))
    down = fr.to_bf16((rng.standard_normal((experts, w, f)) / f ** 0.5).astype(np.float32))
    h = np.zeros((rows, wp), np.float32)
    h[:, :w] = fr.to_bf16(rng.standard_normal((rows, w)).astype(np.float32))
    z = rng.standard_normal((rows, experts)).astype(np.float32)
    z[:, 0] += 1.0   # unequal shares
    dt = torch.bfloat16 if bf16 else torch.float32
    pair, _, tiles, n_tiles, srt, most = ops.moe_route(experts, top, 1, 1, tile, _dev(z, cuda), _dev(h, cuda, dt))
    gu, dn = np.zeros((experts, 2 * fp, wp), np.float32), np.zeros((experts, wp, fp), np.float32)
    gu[:, :, :w], dn[:, :w, :f] = _interleave(gate, up), down
    status = torch.zeros(1, dtype=torch.int32, device=cuda)
    kw = dict(tiles=tiles, n_tiles=n_tiles, max_tiles=most, tile_rows=tile, batch=experts)
    if bf16:
        a = ops.dense_bf16(srt, _dev(gu, cuda, dt), rows * top, 2 * fp, wp, swiglu=1, status=status, **kw)
        y = ops.dense_bf16(a, _dev(dn, cuda, dt), rows * top, wp, fp, out_f32=True, status=status, **kw)
    else:
        t = ops.dense_f32(srt, _dev(gu.transpose(0, 2, 1), cuda), rows * top, 2 * fp, wp, **kw)
        a = ops.gated_pairs_f32(t, fp)
        y = ops.dense_f32(a, _dev(dn.transpose(0, 2, 1), cuda), rows * top, wp, fp, **kw)
    assert int(status) == 0
    pair, a, y = pair.cpu().numpy(), a.float().cpu().numpy(), y.cpu().numpy()
    for r in range(0, rows, max(1, rows // 60)):
        chosen, _ = fr.route(z[r].astype(float), top, 1, 1)
        for k, e in enumerate(chosen):
            mid = fr.silu(h[r, :w].astype(float) @ gate[e].T) * (h[r, :w].astype(float) @ up[e].T)
            want = mid @ down[e].T
            tol = (2e-2 if bf16 else 1e-5) * max(1.0, np.abs(want).max())
            assert np.abs(a[pair[r, k], :f] - mid).max() < (2 ** -7 * np.abs(mid).max() + 1e-3 if bf16 else 1e-5), (r, k)
            assert np.abs(y[pair[r, k], :w] - want).max() < tol, (r, k)
            assert (a[pair[r, k], f:] == 0).all()


# ---- attention ---------------------------------------------------------------------------------------------------------
class _Cache:
    """Sequences of given lengths in scattered pages; projection rows on the device and on the host (in float64)."""

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

    def rows(self, q, k, v):
        """[n][H][dim], [n][G][dim], [n][G][vdim] -> projection rows, appended to the cache."""
        a, n = self.a, q.shape[0]
        row = np.zeros((n, a.q_row), np.float32)
        for x, off, st, w in ((q, 0, a.q_head_stride, a.dim), (k, a.k_offset, a.k_head_stride, a.dim), (v, a.v_offset, a.v_head_stride, a.vdim)):
            for h in range(x.shape[1]):
                row[:, off + h * st:off + h * st + w] = x[:, h]
        d = _dev(row, self.cuda, self.dt)
        ops.grouped_append(a, d, _i32(self.pos, self.cuda), _i32(self.slot, self.cuda), self.table, self.pool)
        return d

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

    def attend(self, d, slot, pos, r1, r2, mode, splits):
        f = lambda r: None if r is None else _dev(np.asarray(r, np.float32), self.cuda)  # noqa: E731
        got, status = ops.grouped_attention(self.a, d, self.pool, self.table, _i32(slot, self.cuda), _i32([p + 1 for p in pos], self.cuda), max(pos) + 1, f(r1), f(r2),
                                            tiles=self.tiles(slot, pos) if mode == "tc" else None, splits=splits if mode == "tc" else 1)
        assert int(status) == 0
        return got.float().cpu().numpy()[:, :, :self.a.vdim]


def _first(a, i):
    return {gm.MASK_CAUSAL: 0, gm.MASK_WINDOW: max(0, i - a.mask_size + 1), gm.MASK_CHUNK: i // max(a.mask_size, 1) * max(a.mask_size, 1)}[a.mask]


def _attend(a, q, k, v, pos, r1, r2):
    """Queries q [n][H][dim] at `pos` over the keys and values of one sequence -> [n][H][vdim], scores' weights."""
    group = a.heads // a.kv_heads
    out = np.zeros((len(pos), a.heads, a.vdim))
    for n, i in enumerate(pos):
        lo = _first(a, i)
        for h in range(a.heads):
            s = k[lo:i + 1, h // group] @ q[n, h] * a.scale
            if a.softcap:
                s = fr.soft_cap(s, a.softcap)
            if r1 is not None:
                s = s - fr.distance_penalty(r1[h], r2[h], i - np.arange(lo, i + 1))
            p = np.exp(s - s.max())
            out[n, h] = (p / p.sum()) @ v[lo:i + 1, h // group]
    return out


SHAPES = [  # heads, kv heads, dim, vdim, mask, size, soft cap, penalty
    (1, 1, 8, 8, 2, 1, 5.0, True), (6, 2, 24, 40, 2, 9, 12.0, True), (4, 4, 96, 72, 2, 63, 30.0, True), (16, 2, 64, 128, 2, 64, 0.0, True),
    (5, 1, 40, 20, 1, 65, 8.0, False), (32, 4, 128, 128, 2, 200, 50.0, True), (12, 3, 192, 256, 0, 0, 20.0, True), (130, 1, 8, 16, 2, 31, 4.0, True),
    (2, 1, 272, 320, 2, 50, 9.0, True), (7, 7, 13, 5, 2, 17, 3.0, True), (40, 8, 80, 48, 0, 0, 0.0, False)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
def test_grouped_attention_prompt(cuda, shape, mode):
    heads, kv, dim, vdim, mask, size, cap, penalty = shape
    a = ops.grouped_layout(heads, kv, dim, vdim, mask, size, 1.7 * dim ** -0.5, cap, penalty, bf16=mode != "f32")
    if mode == "tc" and ops.grouped_tile_tokens(a) == 0:
        assert vdim > 256 or dim > 256
        pytest.skip("these sizes belong to the plain kernel")
    rng = np.random.default_rng(dim + size)
    lens = [150, 1, 37, 16]
    c = _Cache(rng, cuda, a, lens)
    n = sum(lens)
    q, k, v = (fr.to_bf16(rng.standard_normal((n, g, w)).astype(np.float32)) for g, w in ((heads, dim), (kv, dim), (kv, vdim)))
    r1, r2 = (rng.uniform(0.1, 1.5, heads).astype(np.float32), rng.uniform(0.02, 2.0, heads).astype(np.float32)) if penalty else (None, None)
    d = c.rows(q, k, v)
    want, o = [], 0
    for m in lens:
        want.append(_attend(a, q[o:o + m].astype(float), k[o:o + m].astype(float), v[o:o + m].astype(float), range(m), r1, r2))
        o += m
    want = np.concatenate(want)
    for splits in ((1, 2, 5) if mode == "tc" else (1,)):
        got = c.attend(d, c.slot, c.pos, r1, r2, mode, splits)
        assert np.abs(got - want).max() < (1e-5 if mode == "f32" else 2 ** -8 * np.abs(want).max() + 1e-3), splits


@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("mask,size", [(2, 1), (2, 15), (2, 16), (2, 17), (2, 64), (2, 100), (2, 128), (2, 1000), (1, 1), (1, 17), (1, 64), (1, 130), (0, 0)])
@pytest.mark.parametrize("as_prompt", [False, True])
def test_grouped_attention_sees_exactly_the_mask(cuda, mode, mask, size, as_prompt):
    """One stored key points along the query and outweighs all others: the output is its value while the mask lets it through and has
    no trace of it otherwise; just inside and outside every edge, at page borders and past the first block of keys."""
    heads, kv, dim, vdim, n = 6, 2, 40, 24, 450
    a = ops.grouped_layout(heads, kv, dim, vdim, mask, size, 1.0, 0.0, True, bf16=mode != "f32")
    rng = np.random.default_rng(size)
    c = _Cache(rng, cuda, a, [n])
    q, k, v = (fr.to_bf16(rng.standard_normal((n, g, w)).astype(np.float32)) for g, w in ((heads, dim), (kv, dim), (kv, vdim)))
    r1, r2 = np.full(heads, 0.2, np.float32), np.full(heads, 0.5, np.float32)
    c.rows(q, k, v)
    for far in (0, 1, 15, 16, 17, 47, 48, 63, 64, 128, 200, 207, 208):
        edge = far + size if mask == 1 else (far // size + 1) * size if mask == 2 else n   # the first position that does not see it
        at = sorted({p for p in (far, edge - 2, edge - 1, edge, edge + 1) if far <= p < n} | ({n - 1} if mask == 0 else set()))
        if as_prompt:   # one run that crosses the edge
            at = list(range(max(at[0], at[-1] - 30), at[-1] + 1))
        qf = np.zeros((len(at), heads, dim), np.float32)
        for h in range(heads):
            key = k[far, h // 3]
            qf[:, h] = fr.to_bf16(20.0 * key / np.linalg.norm(key))
        row = np.zeros((len(at), a.q_row), np.float32)
        for h in range(heads):
            row[:, h * a.q_head_stride:h * a.q_head_stride + dim] = qf[:, h]
        d = _dev(row, cuda, c.dt)
        want = _attend(a, qf.astype(float), k.astype(float), v.astype(float), at, r1, r2)
        for splits in ((1, 3) if mode == "tc" else (1,)):
            got = c.attend(d, [0] * len(at), at, r1, r2, mode, splits)
            assert np.abs(got - want).max() < (1e-4 if mode == "f32" else 2e-2 * np.abs(want).max()), (far, at, splits)
        for i, p in enumerate(at):   # the spike is where it should be, so that the comparison above means something
            is_far = max(np.abs(want[i, h] - v[far, h // 3]).max() for h in range(heads)) < 0.2
            assert is_far == (far >= _first(a, p)), (far, p)


def test_grouped_decode_equals_prompt_rows(cuda):
    """The same rows as one prompt, as single-token tiles with split keys, and mixed with another sequence's."""
    a = ops.grouped_layout(8, 2, 72, 40, gm.MASK_CHUNK, 170, 0.12, 15.0, True)
    rng = np.random.default_rng(3)
    c = _Cache(rng, cuda, a, [300, 77])
    q, k, v = (fr.to_bf16(rng.standard_normal((377, g, w)).astype(np.float32)) for g, w in ((8, 72), (2, 72), (2, 40)))
    r1, r2 = rng.uniform(0.1, 1.0, 8), rng.uniform(0.1, 1.0, 8)
    d = c.rows(q, k, v)
    whole = c.attend(d, c.slot, c.pos, r1, r2, "tc", 1)
    for pick in ([5], [299, 376], [0, 300, 64, 169, 310, 170, 171, 299]):
        for splits in (1, 2, 3, 4, 9, 40):
            got = c.attend(d[pick].contiguous(), [c.slot[i] for i in pick], [c.pos[i] for i in pick], r1, r2, "tc", splits)
            assert np.abs(got - whole[pick]).max() < 2 ** -7 * np.abs(whole).max()


# ---- delta rule --------------------------------------------------------------------------------------------------------
def _runs(parts, parity, cuda):
    """parts: (slot, first position, rows) of every run -> the row arrays and the first rows of the runs."""
    slot, pos, first, last, par, starts = [], [], [], [], [], []
    for s, p, n in parts:
        r0 = len(slot)
        starts.append(r0)
        for i in range(n):
            slot.append(s), pos.append(p + i), first.append(r0), last.append(r0 + n - 1), par.append(parity[s])
    return tuple(_i32(a, cuda) for a in (slot, pos, first, last, par)), _i32(starts, cuda)


DELTA_SHAPES = [  # heads, q/k heads, dim, vdim, taps, decay rank, gate rank
    (1, 1, 8, 8, 4, 8, 8), (4, 2, 16, 24, 3, 10, 6), (6, 6, 32, 64, 4, 24, 40), (3, 1, 5, 7, 2, 3, 1), (2, 2, 64, 40, 1, 8, 8), (4, 4, 128, 128, 4, 16, 16),
    (2, 1, 100, 130, 5, 16, 16), (2, 2, 200, 260, 4, 8, 8), (1, 1, 300, 33, 7, 8, 8),
    (16, 8, 40, 24, 4, 8, 8), (30, 10, 40, 24, 4, 8, 8)]   # columns per warp depend on the number of heads and runs


@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("bf16", [False, True])
def test_delta_rule_carries_its_states_over_any_cut(cuda, shape, bf16):
    heads, kv, dim, vdim, taps, dr, gr = shape
    rng = np.random.default_rng(dim + vdim)
    a = ops.delta_layout(heads, kv, dim, vdim, taps, dr, gr, 1e-5, bf16=bf16)
    n, dt = 70, torch.bfloat16 if bf16 else torch.float32
    rnd = lambda x: fr.to_bf16(x.astype(np.float32)) if bf16 else x.astype(np.float32)  # noqa: E731
    ch = 2 * kv * dim + heads * vdim
    conv = (0.5 * rng.standard_normal((ch, taps))).astype(np.float32)
    a_log, dt_bias = np.log(rng.uniform(0.3, 3.0, heads)).astype(np.float32), rng.uniform(-6, 0, heads * dim).astype(np.float32)
    norm = (1 + 0.3 * rng.standard_normal(vdim)).astype(np.float32)
    raw = rnd(rng.standard_normal((3, n, ch)))
    raw[:, 40, :2 * kv * dim] *= 8.0     # keys that stand out
    beta = rnd(rng.standard_normal((3, n, heads)))
    dec, gate = rng.standard_normal((3, n, heads * dim)).astype(np.float32), rnd(rng.standard_normal((3, n, heads * vdim)))
    raw, beta, gate = (rnd(x) for x in (raw, beta, gate))
    of = np.arange(heads) // (heads // kv)
    want = []
    for s in range(3):
        x = fr.silu(fr.short_conv(raw[s].astype(float), conv.astype(float)))
        q = (fr.unit(x[:, :kv * dim].reshape(n, kv, dim)) * dim ** -0.5)[:, of]
        k = fr.unit(x[:, kv * dim:2 * kv * dim].reshape(n, kv, dim))[:, of]
        g = fr.channel_decay(dec[s].astype(float).reshape(n, heads, dim), a_log.astype(float), dt_bias.astype(float).reshape(heads, dim))
        o = fr.delta_rule(q, k, x[:, 2 * kv * dim:].reshape(n, heads, vdim), g, fr.sigmoid(beta[s].astype(float)))
        want.append(fr.rms(o, 1e-5) * norm * fr.sigmoid(gate[s].astype(float).reshape(n, heads, vdim)))

    def proj(s, lo, hi):
        row = np.full((hi - lo, a.row), 7.0, np.float32)
        for off, x in ((a.q_offset, raw[s, lo:hi, :kv * dim]), (a.k_offset, raw[s, lo:hi, kv * dim:2 * kv * dim]), (a.v_offset, raw[s, lo:hi, 2 * kv * dim:]),
                       (a.beta_offset, beta[s, lo:hi])):
            row[:, off:off + x.shape[1]] = x
        return row

    def padded(x, width):
        return np.concatenate([x, np.full((x.shape[0], width - x.shape[1]), 5.0, np.float32)], axis=1)

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
            cat = lambda f: np.concatenate([f(s, p, p + m) for s, p, m in parts])  # noqa: E731
            runs, starts = _runs(parts, parity, cuda)
            got = ops.delta_rule(a, _dev(cat(proj), cuda, dt), _dev(padded(cat(lambda s, l, h: dec[s, l:h]), a.decay_row), cuda),
                                 _dev(padded(cat(lambda s, l, h: gate[s, l:h]), a.gate_row), cuda, dt), *consts, state, conv_state, runs, starts)
            w = cat(lambda s, l, h: want[s][l:h])
            g = got.float().cpu().numpy()
            tol = 2 ** -8 * np.abs(w).max() + 1e-4 if bf16 else 5e-5 * max(1.0, np.abs(w).max())
            assert np.abs(g[:, :, :vdim] - w).max() < tol, (cuts, parts)
            assert (g[:, :, vdim:] == 0).all()
            for s, p, m in parts:
                at[s] += m
                parity[s] ^= 1
