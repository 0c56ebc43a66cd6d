"""The mechanisms of the layered models one by one, each through the C ABI against a plain reference of the same equation:
dense matmuls (strides, batches, xIELU, soft cap), the output norm + residual + short convolution with its state, the latent
append and the two latent attention kernels (window edges, splits, far keys)."""
import numpy as np
import pytest
import torch

from gptrs_b200 import ops
from oracle import bevosun_ref as br

pytestmark = pytest.mark.gpu


def _dev(a, cuda, dt=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).to(cuda)
    return t if dt is None else t.to(dt)


def _i32(a, cuda):
    return torch.tensor(list(a), dtype=torch.int32, device=cuda)


# ---- dense matmuls -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (3, 72, 40), (16, 264, 136), (17, 128, 64), (33, 1000, 320), (64, 136, 2048), (65, 384, 104), (128, 256, 72),
                                   (129, 8, 24), (200, 72, 200), (700, 264, 328), (1500, 3072, 256)])
def test_dense_bf16(cuda, m, n, k):
    g = torch.Generator(device=cuda).manual_seed(m + n + k)
    x = torch.randn(m, k, device=cuda, generator=g).bfloat16()
    w = (torch.randn(n, k, device=cuda, generator=g) / k ** 0.5).bfloat16()
    b = torch.randn(n, device=cuda, generator=g)
    z = (x.double() @ w.double().T + b.double()).cpu().numpy()
    got = ops.dense_bf16(x, w, m, n, k, bias=b, out_f32=True).cpu().numpy()
    assert np.abs(got - z).max() < 1e-4
    got = ops.dense_bf16(x, w, m, n, k, bias=b).float().cpu().numpy()
    assert np.abs(got - z).max() < 2 ** -8 * np.abs(z).max()
    p, q = 0.3, -0.7
    pair = (float(br.softplus(p)), 0.5 + float(br.softplus(q)))
    want = br.xielu(z, p, q)
    got = ops.dense_bf16(x, w, m, n, k, bias=b, xielu=pair).float().cpu().numpy()
    assert np.abs(got - want).max() < 2 ** -8 * np.abs(want).max() + 1e-4
    got = ops.dense_bf16(x, w, m, n, k, bias=b, out_f32=True, softcap=1.5).cpu().numpy()
    assert np.abs(got - br.soft_cap(z, 1.5)).max() < 1e-4


@pytest.mark.parametrize("m", [1, 9, 40, 70, 128, 150, 400])
@pytest.mark.parametrize("heads,n,k,gap", [(5, 24, 16, 8), (3, 200, 72, 64), (2, 64, 136, 16)])
def test_dense_bf16_batches_with_strides(cuda, m, heads, n, k, gap):
    g = torch.Generator(device=cuda).manual_seed(m)
    x = torch.randn(m, heads, k + gap, device=cuda, generator=g).bfloat16()
    w = (torch.randn(heads, n, k, device=cuda, generator=g) / k ** 0.5).bfloat16()
    y = torch.full((m, heads, n + gap), 7.0, device=cuda, dtype=torch.bfloat16)
    ops.dense_bf16(x, w, m, n, k, out=y, ldx=heads * (k + gap), ldy=heads * (n + gap), batch=heads, x_step=k + gap, y_step=n + gap)
    want = torch.einsum("mhk,hnk->mhn", x[:, :, :k].double(), w.double())
    assert (y[:, :, :n].double() - want).abs().max() < 2 ** -8 * want.abs().max()
    assert (y[:, :, n:] == 7.0).all()   # columns between the batches are left alone


def test_dense_f32_batches_with_strides(cuda):
    g = torch.Generator(device=cuda).manual_seed(0)
    for m, heads, n, k in ((1, 3, 20, 13), (2, 1, 300, 64), (11, 4, 9, 50), (37, 2, 130, 7)):
        x = torch.randn(m, heads, k + 3, device=cuda, generator=g)
        w = torch.randn(heads, k, n, device=cuda, generator=g)
        b = torch.randn(n, device=cuda, generator=g)
        y = torch.full((m, heads, n + 1), 7.0, device=cuda)
        ops.dense_f32(x, w, m, n, k, out=y, bias=b, xielu=(0.9, 1.1), softcap=5.0, ldx=heads * (k + 3), ldy=heads * (n + 1), batch=heads, x_step=k + 3, y_step=n + 1)
        z = torch.einsum("mhk,hkn->mhn", x[:, :, :k].double(), w.double()).cpu().numpy() + b.double().cpu().numpy()
        a = np.where(z > 0, 0.9 * z * z + z / 2, 1.1 * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0)) + z / 2)
        assert np.abs(y[:, :, :n].cpu().numpy() - br.soft_cap(a, 5.0)).max() < 2e-5
        assert (y[:, :, n:] == 7.0).all()


@pytest.mark.parametrize("m", [1, 20, 100, 128])
def test_greedy_candidates_of_the_dense_head(cuda, m):
    g = torch.Generator(device=cuda).manual_seed(m)
    n, k = 520, 64
    x = torch.randn(m, k, device=cuda, generator=g).bfloat16()
    w = torch.randn(n, k, device=cuda, generator=g).bfloat16()
    tiles = (n + 127) // 128
    best = (torch.zeros(tiles, m, device=cuda), torch.zeros(tiles, m, dtype=torch.int32, device=cuda))
    logits = ops.dense_bf16(x, w, m, n, k, out_f32=True, softcap=30.0)
    ops.dense_bf16(x, w, m, n, k, out=torch.empty_like(logits), out_f32=True, softcap=30.0, best=best)
    assert torch.equal(ops.pick_best(*best).long(), logits.argmax(dim=1))


def test_dense_bf16_refuses_unaligned_sizes(cuda):
    x = torch.zeros(4, 64, device=cuda, dtype=torch.bfloat16)
    for n, k in ((12, 64), (16, 60)):
        with pytest.raises(Exception, match="multiples of 8"):
            ops.dense_bf16(x, x, 4, n, k)


# ---- output norm + residual + short convolution ------------------------------------------------------------------------
def _runs(parts, parity, cuda):
    """parts: (slot, first position, rows) of every run -> the five row arrays."""
    slot, pos, first, last, par = [], [], [], [], []
    for s, p, n in parts:
        r0 = len(slot)
        for i in range(n):
            slot.append(s), pos.append(p + i), first.append(r0), last.append(r0 + n - 1), par.append(parity[s])
    return tuple(_i32(a, cuda) for a in (slot, pos, first, last, par))


@pytest.mark.parametrize("dim,taps", [(40, 3), (37, 4), (256, 2), (1032, 3), (24, 1), (30, 7), (64, 16)])
@pytest.mark.parametrize("big", [False, True])
def test_conv_step_carries_the_state_over_any_cut(cuda, dim, taps, big):
    rng = np.random.default_rng(dim + taps)
    n = 1300 if big else 60
    conv = rng.standard_normal((dim, taps)).astype(np.float32)
    gamma = (1 + 0.3 * rng.standard_normal(dim)).astype(np.float32)
    xs = [rng.standard_normal((n, dim)).astype(np.float32) for _ in range(3)]
    ys = [rng.standard_normal((n, dim)).astype(np.float32) for _ in range(3)]
    want_x = [x + br.rms_norm(y.astype(float), gamma, 1e-4) for x, y in zip(xs, ys)]
    want_h = [br.conv_input(x, conv.astype(float)) for x in want_x]
    state = torch.full((3, 2, max(taps - 1, 1), dim), 9.0, device=cuda)   # what a slot's last user left must not show
    parity, at = [0, 1, 0], [0, 0, 0]
    cuts = [1, 2, 1, 1, 3, 19, 2, 1, 400, 1, 5, 700] if big else [1, 2, 1, 1, 3, 19, 2, 1]
    i = 0
    while min(at) < n:
        parts = []
        for s in rng.permutation(3):
            c = min(cuts[i % len(cuts)], n - at[s])
            i += 1
            if c > 0 and rng.random() < 0.8:
                parts.append((int(s), at[s], c))
        if not parts:
            continue
        x = np.concatenate([xs[s][p:p + c] for s, p, c in parts])
        y = np.concatenate([ys[s][p:p + c] for s, p, c in parts])
        gx, gh = ops.post_norm_conv(_dev(gamma, cuda), 1e-4, len(x), dim, x=_dev(x, cuda), y=_dev(y, cuda), conv=_dev(conv, cuda), state=state,
                                    runs=_runs(parts, parity, cuda))
        assert np.abs(gx.cpu().numpy() - np.concatenate([want_x[s][p:p + c] for s, p, c in parts])).max() < 1e-5
        assert np.abs(gh.cpu().numpy() - np.concatenate([want_h[s][p:p + c] for s, p, c in parts])).max() < 1e-4
        for s, p, c in parts:
            at[s] += c
            parity[s] ^= 1


def test_conv_step_embedding_and_bf16(cuda):
    rng = np.random.default_rng(0)
    v, d, n = 50, 36, 33
    embed, gamma = rng.standard_normal((v, d)).astype(np.float32), (1 + 0.3 * rng.standard_normal(d)).astype(np.float32)
    conv = rng.standard_normal((d, 3)).astype(np.float32)
    tok = rng.integers(0, v, n)
    x = br.rms_norm(embed[tok].astype(float), gamma, 1e-5)
    state = torch.zeros(1, 2, 2, d, device=cuda)
    gx, gh = ops.post_norm_conv(_dev(gamma, cuda), 1e-5, n, d, embed=_dev(embed, cuda), tokens=_i32(tok, cuda), conv=_dev(conv, cuda), state=state,
                                runs=_runs([(0, 0, n)], [0], cuda), out_dtype=torch.bfloat16, ldh=40)
    h = br.conv_input(x, conv.astype(float))
    assert np.abs(gx.cpu().numpy() - x).max() < 1e-5
    assert np.abs(gh[:, :d].float().cpu().numpy() - h).max() < 2 ** -8 * np.abs(h).max() and (gh[:, d:] == 0).all()
    status = torch.zeros(1, dtype=torch.int32, device=cuda)
    tok[5] = v   # out of range: flagged, nothing read outside the table
    ops.post_norm_conv(_dev(gamma, cuda), 1e-5, n, d, embed=_dev(embed, cuda), tokens=_i32(tok, cuda), status=status)
    assert int(status) == 2


def test_post_norm_final(cuda):
    rng = np.random.default_rng(1)
    x, y = rng.standard_normal((9, 70)).astype(np.float32), rng.standard_normal((9, 70)).astype(np.float32)
    g, f = (1 + 0.2 * rng.standard_normal((2, 70))).astype(np.float32)
    want = br.rms_norm(x + br.rms_norm(y.astype(float), g, 1e-3), f, 1e-3)
    for rows in (None, [8, 0, 0, 5]):
        got = ops.post_norm_final(_dev(x, cuda), _dev(y, cuda), _dev(g, cuda), _dev(f, cuda), 1e-3, rows=None if rows is None else _i32(rows, cuda))
        assert np.abs(got.cpu().numpy() - (want if rows is None else want[rows])).max() < 1e-5


# ---- latent attention --------------------------------------------------------------------------------------------------
class _Cache:
    """Sequences of given lengths in scattered pages; what the kernels should read is kept on the host in float64."""

    def __init__(self, rng, cuda, a, bf16, lens, base=100.0):
        self.a, self.bf16, self.cuda, self.lens = a, bf16, cuda, lens
        self.dt = torch.bfloat16 if bf16 else torch.float32
        self.pages = [(n + 15) // 16 for n in lens]
        self.max_pages = max(self.pages) + 1
        total = sum(self.pages) + 3
        perm = rng.permutation(total)
        table = np.zeros((len(lens), self.max_pages), np.int32)
        o = 0
        for s, n in enumerate(self.pages):
            table[s, :n] = perm[o:o + n]
            o += n
        self.table = _dev(table, cuda)
        # rows that nobody has written are poison: a result that touches one is not a number
        self.pool = torch.full((total * a.page_bytes // (2 if bf16 else 4),), float("nan"), device=cuda, dtype=self.dt)
        self.norm_w = br.to_bf16((1 + 0.2 * rng.standard_normal(a.kv_rank)).astype(np.float32))
        half, n_pos = a.rot_dims // 2, max(lens) + 1
        ang = np.arange(n_pos)[:, None] * base ** (-2.0 * np.arange(half) / max(a.rot_dims, 1))
        self.cos, self.sin, self.base = np.cos(ang).astype(np.float32), np.sin(ang).astype(np.float32), base

    def append(self, rng, slot, pos):
        """Random projection rows for (slot, pos): the absorbed queries on the device, queries and cache rows on the host."""
        a, n = self.a, len(slot)
        qkv = np.zeros((n, a.q_row), np.float32)
        cols = [h * a.q_head_stride + a.q_rot_offset + c for h in range(a.heads) for c in range(a.rot_dim)]
        qkv[:, cols] = rng.standard_normal((n, len(cols)))
        qkv[:, a.dkv_offset:a.dkv_offset + a.kv_rank] = rng.standard_normal((n, a.kv_rank))
        qkv[:, a.rot_offset:a.rot_offset + a.rot_dim] = rng.standard_normal((n, a.rot_dim))
        qa = np.full((n, a.heads, a.qa_head_stride), 0.0, np.float32)
        qa[:, :, :a.kv_rank] = rng.standard_normal((n, a.heads, a.kv_rank))
        if self.bf16:
            qkv, qa = br.to_bf16(qkv), br.to_bf16(qa)
        d_qa = _dev(qa, self.cuda, self.dt)
        ops.latent_append(a, _dev(qkv, self.cuda, self.dt), _i32(pos, self.cuda), _i32(slot, self.cuda), self.table, _dev(self.norm_w, self.cuda), 1e-5,
                          _dev(self.cos, self.cuda), _dev(self.sin, self.cuda), d_qa, self.pool)
        lat = br.rms_norm(qkv[:, a.dkv_offset:a.dkv_offset + a.kv_rank].astype(float), self.norm_w, 1e-5)
        k_rot = br.rotate_interleaved(qkv[:, a.rot_offset:a.rot_offset + a.rot_dim].astype(float), pos, self.base, a.rot_dims)
        q_rot = br.rotate_interleaved(qkv[:, cols].astype(float).reshape(n, a.heads, a.rot_dim), pos, self.base, a.rot_dims)
        rows = np.concatenate([lat, k_rot], axis=1)
        q = np.concatenate([qa[:, :, :a.kv_rank].astype(float), q_rot], axis=2)
        if self.bf16:
            rows, q = br.to_bf16(rows.astype(np.float32)).astype(float), br.to_bf16(q.astype(np.float32)).astype(float)
        return d_qa, q, rows

    def tiles(self, slot, pos):
        t = ops.latent_tile_tokens(self.a)
        first, count, i, n = [], [], 0, len(slot)
        while i < n:
            e = i + 1
            while e < n and e - i < t and slot[e] == slot[i] and pos[e] == pos[e - 1] + 1:
                e += 1
            first.append(i), count.append(e - i)
            i = e
        return _i32(first, self.cuda), _i32(count, self.cuda)


def _attend(q, rows, pos, a):
    """q [n][H][rank + rot], rows of one sequence, positions of the queries -> [n][H][rank]."""
    out = np.zeros((len(pos), a.heads, a.kv_rank))
    for i, p in enumerate(pos):
        lo = max(0, p - a.window + 1)
        s = q[i] @ rows[lo:p + 1].T * a.scale
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = (w / w.sum(axis=1, keepdims=True)) @ rows[lo:p + 1, :a.kv_rank]
    return out


SHAPES = [  # heads, dim, rot, vdim, rank, window
    (1, 8, 2, 8, 8, 1), (3, 24, 12, 20, 40, 9), (7, 16, 16, 24, 72, 63), (16, 32, 8, 16, 120, 64), (5, 40, 80, 8, 64, 65), (40, 16, 32, 16, 256, 200),
    (64, 8, 64, 8, 200, 1000), (130, 8, 8, 8, 56, 31), (4, 16, 16, 16, 300, 50), (2, 8, 20, 8, 180, 17)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
def test_latent_attention_prompt(cuda, shape, mode):
    heads, dim, rot, vdim, rank, window = shape
    bf16 = mode != "f32"
    a = ops.latent_layout(heads, dim, rot, vdim, rank, window, 1.3 * (rank + rot) ** -0.5, bf16=bf16)
    if mode == "tc" and ops.latent_tile_tokens(a) == 0:
        assert rank > 256
        pytest.skip("these sizes belong to the plain kernel")
    rng = np.random.default_rng(rank + window)
    lens = [150, 1, 37, 16]
    c = _Cache(rng, cuda, a, bf16, lens)
    slot = [s for s, n in enumerate(lens) for _ in range(n)]
    pos = [p for n in lens for p in range(n)]
    d_qa, q, rows = c.append(rng, slot, pos)
    for splits in ((1, 2, 5) if mode == "tc" else (1,)):
        got, status = ops.latent_attention(a, d_qa, c.pool, c.table, _i32(slot, cuda), _i32([p + 1 for p in pos], cuda), max(lens),
                                           tiles=c.tiles(slot, pos) if mode == "tc" else None, splits=splits)
        assert int(status) == 0
        got, o = got.float().cpu().numpy(), 0
        for n in lens:
            want = _attend(q[o:o + n], rows[o:o + n], range(n), a)
            assert np.abs(got[o:o + n, :, :rank] - want).max() < (1e-5 if mode == "f32" else 2 ** -8 * np.abs(want).max() + 2e-3), (splits, n)
            o += n


@pytest.mark.parametrize("mode", ["f32", "bf16", "tc"])
@pytest.mark.parametrize("window", [1, 15, 16, 17, 64, 100, 128, 1000])
@pytest.mark.parametrize("as_prompt", [False, True])
def test_latent_attention_sees_exactly_the_window(cuda, mode, window, as_prompt):
    """One stored latent points along the query and outweighs all others: the output is that latent while it is inside the
    window (itself and window - 1 before) and has no trace of it one token later; at page borders and past the first block."""
    bf16 = mode != "f32"
    heads, rank, rot = 3, 40, 8
    a = ops.latent_layout(heads, 16, rot, 16, rank, window, 1.0, bf16=bf16)
    rng = np.random.default_rng(window)
    n = 450
    c = _Cache(rng, cuda, a, bf16, [n])
    d_qa, q, rows = c.append(rng, [0] * n, list(range(n)))
    pool_rows = rows.copy()
    for far in (0, 1, 15, 16, 17, 47, 48, 63, 64, 128, 200, 207, 208):
        at = [p for p in (far, far + window - 2, far + window - 1, far + window, far + window + 1) if far <= p < n]
        if as_prompt:   # one run that crosses the edge
            at = list(range(max(at[0], at[-1] - 30), at[-1] + 1))
        qf = np.zeros((len(at), heads, a.qa_head_stride), np.float32)
        unit = pool_rows[far, :rank] / np.linalg.norm(pool_rows[far, :rank])
        qf[:, :, :rank] = br.to_bf16((20.0 * unit).astype(np.float32))
        qd = _dev(qf, cuda, c.dt)
        tiles = c.tiles([0] * len(at), at) if mode == "tc" else None
        for splits in ((1, 3) if mode == "tc" else (1,)):
            got, status = ops.latent_attention(a, qd, c.pool, c.table, _i32([0] * len(at), cuda), _i32([p + 1 for p in at], cuda), n, tiles=tiles, splits=splits)
            assert int(status) == 0
            q_host = np.concatenate([qf[:, :, :rank], np.zeros((len(at), heads, rot))], axis=2)
            want = _attend(q_host, pool_rows, at, a)
            got = got.float().cpu().numpy()[:, :, :rank]
            assert np.abs(got - want).max() < (1e-4 if mode == "f32" else 2e-2 * np.abs(want).max()), (far, at, splits)
            for i, p in enumerate(at):   # the spike is where it should be, so that the comparison above means something
                is_far = np.abs(want[i] - pool_rows[far, :rank]).max() < 0.2
                assert is_far == (p - far < window), (far, p)


def test_latent_decode_equals_prompt_rows(cuda):
    """The same rows as one prompt, as single-token tiles with split keys, and mixed with another sequence's."""
    a = ops.latent_layout(8, 16, 16, 16, 96, 130, 0.1)
    rng = np.random.default_rng(3)
    lens = [300, 77]
    c = _Cache(rng, cuda, a, True, lens)
    slot = [0] * 300 + [1] * 77
    pos = list(range(300)) + list(range(77))
    d_qa, q, rows = c.append(rng, slot, pos)
    ctx = [p + 1 for p in pos]
    whole, _ = ops.latent_attention(a, d_qa, c.pool, c.table, _i32(slot, cuda), _i32(ctx, cuda), 300, tiles=c.tiles(slot, pos), splits=1)
    for pick in ([5], [299, 376], [0, 300, 64, 200, 310, 129, 130, 131]):
        sl, ps = [slot[i] for i in pick], [pos[i] for i in pick]
        for splits in (1, 2, 3, 4, 9):
            got, status = ops.latent_attention(a, d_qa[pick].contiguous(), c.pool, c.table, _i32(sl, cuda), _i32([p + 1 for p in ps], cuda), 300,
                                               tiles=(_i32(range(len(pick)), cuda), _i32([1] * len(pick), cuda)), splits=splits)
            assert int(status) == 0
            assert (got.float() - whole[pick].float()).abs().max() < 2 ** -7 * whole.float().abs().max()
