"""The bf16-weight layers one by one (lbk_sandwich_norm, lbk_dense_linear, lbk_attn_window, lbk_moe_route) against the
plain numpy functions of the Pefolix oracle, in both compute types, at sizes that are not multiples of anything."""
import numpy as np
import pytest

pytestmark = pytest.mark.gpu
BF16, F32 = 0, 1


@pytest.fixture(scope="module")
def po():
    from oracle import pefolix_oracle
    return pefolix_oracle


def _lib():
    from lemonade_burn_b200 import _lib as L
    return L, L.load()


def _st():
    import torch
    return torch.cuda.current_stream().cuda_stream


def pad64(n):
    return (n + 63) // 64 * 64


def dev_rows(a, compute, pitch=None):
    """numpy [m, n] -> device rows of the compute type with zeros up to `pitch`; returns (tensor, exact values)."""
    import torch
    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32))
    t = t.to(torch.bfloat16) if compute == BF16 else t
    out = torch.zeros(a.shape[0], pitch or a.shape[1], dtype=t.dtype)
    out[:, :a.shape[1]] = t
    return out.cuda(), t.double().numpy()


@pytest.mark.parametrize("n", [4, 72, 250, 256, 1000, 2052, 4096, 8192, 8190, 9001])
def test_sandwich_norm(ctx, po, n):
    """x += norm(y) * w_post, then norm(x) * w: rows with a mean far from zero (a norm without the mean would show),
    widths of whole and of ragged 16-byte units, one row and several; f32 and bf16 outputs."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(n)
    for rows, with_y in ((1, True), (5, True), (3, False)):
        x = (rng.standard_normal((rows, n)) + 3.0).astype(np.float32)
        y = (2.0 * rng.standard_normal((rows, n)) - 20.0).astype(np.float32)
        wp, w = (rng.standard_normal(n).astype(np.float32) for _ in range(2))
        eps = 1e-3
        xd, yd, wpd, wd = (torch.from_numpy(a).cuda() for a in (x, y, wp, w))
        of = torch.zeros(rows, n, device="cuda")
        pitch = pad64(n)
        oe = torch.zeros(rows, pitch, dtype=torch.bfloat16, device="cuda")
        L.check(lib.lbk_sandwich_norm(ctx.handle, xd.data_ptr(), yd.data_ptr() if with_y else None, wpd.data_ptr() if with_y else None,
                                      wd.data_ptr(), rows, n, eps, of.data_ptr(), oe.data_ptr(), pitch, _st()))
        want_x = x.astype(np.float64) + (po.layer_norm(y.astype(np.float64), wp, eps) if with_y else 0.0)
        want = po.layer_norm(want_x, w, eps)
        assert np.abs(xd.cpu().numpy() - want_x).max() < 2e-5 * np.abs(want_x).max()
        assert np.abs(of.cpu().numpy() - want).max() < 3e-5 * np.abs(want).max()
        assert np.abs(oe.float().cpu().numpy()[:, :n] - want).max() < 2.0 ** -8 * np.abs(want).max()
        assert not oe[:, n:].any()
    ctx.check_device_error()


DENSE_SHAPES = [(40, 72), (1, 64), (130, 200), (640, 256), (384, 1088), (97, 40)]


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("rows,cols", DENSE_SHAPES)
def test_dense_linear(ctx, po, compute, rows, cols):
    """Plain, squared-relu and gated projections at token counts on both sides of every kernel's limits."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(rows + cols)
    for m in (1, 2, 3, 8, 9, 16, 17, 63, 130, 300):
        x, xv = dev_rows(rng.standard_normal((m, cols)), compute, pad64(cols))
        for gated, relu2, f32 in ((0, 0, 1), (0, 1, 0), (1, 0, 0)):
            w, wv = dev_rows(rng.standard_normal((rows * (2 if gated else 1), cols)) * cols ** -0.5, BF16, pad64(cols))
            pitch = pad64(rows)
            out = torch.full((m, pitch), 7.0, dtype=torch.float32 if (f32 or compute == F32) else torch.bfloat16, device="cuda")
            L.check(lib.lbk_dense_linear(ctx.handle, compute, x.data_ptr(), x.shape[1], m, w.data_ptr(), w.shape[1], w.shape[0], cols, gated,
                                         rows, relu2, out.data_ptr(), pitch, f32, None, 0, _st()))
            v = xv @ wv.T
            want = po.gelu_tanh(v[:, :rows]) * v[:, rows:] if gated else (po.relu2(v) if relu2 else v)
            got = out.float().cpu().numpy()
            tol = 1e-5 if out.dtype == torch.float32 else 2.0 ** -8
            assert np.abs(got[:, :rows] - want).max() <= tol * max(1.0, np.abs(want).max()), (m, gated, relu2)
            assert (got[:, rows:] == 7.0).all()
    ctx.check_device_error()


@pytest.mark.parametrize("rows,cols,m,gated", [(5000, 1024, 2053, 0), (2500, 4096, 2053, 1), (2560, 6912, 2048, 0), (300, 4096, 2000, 1), (129, 8192, 40, 0)])
def test_dense_linear_large(ctx, rows, cols, m, gated):
    """Sizes at which the tile shapes change (two weight boxes a tile, K split over a cluster), ragged in rows and tokens,
    against a 32-bit product of the same values."""
    import torch
    L, lib = _lib()
    torch.manual_seed(rows)
    x = torch.randn(m, cols, device="cuda").to(torch.bfloat16)
    w = (torch.randn(rows * (2 if gated else 1), cols, device="cuda") * cols ** -0.5).to(torch.bfloat16)
    out = torch.full((m, pad64(rows)), 7.0, dtype=torch.bfloat16 if gated else torch.float32, device="cuda")
    L.check(lib.lbk_dense_linear(ctx.handle, BF16, x.data_ptr(), cols, m, w.data_ptr(), cols, w.shape[0], cols, gated, rows, 0, out.data_ptr(),
                                 out.shape[1], 0 if gated else 1, None, 0, _st()))
    v = x.float() @ w.float().T
    want = torch.nn.functional.gelu(v[:, :rows], approximate="tanh") * v[:, rows:] if gated else v
    assert float((out[:, :rows].float() - want).abs().max()) <= (2.0 ** -8 if gated else 2e-5) * float(want.abs().max())
    assert bool((out[:, rows:] == 7.0).all())
    ctx.check_device_error()


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("counts", [[3, 0, 40, 1, 300, 0, 17], [0, 0, 5], [130], [64, 64, 64, 64, 1]])
def test_dense_linear_of_sorted_tokens(ctx, compute, counts):
    """Stacked expert matrices: token rows offs[e] .. offs[e + 1] - 1 meet expert e only; experts without tokens, with
    one, and with several tiles of them."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(sum(counts))
    E, m = len(counts), sum(counts)
    offs = torch.tensor(np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)).cuda()
    for rows, cols in ((72, 40), (200, 256)):
        x, xv = dev_rows(rng.standard_normal((m, cols)), compute, pad64(cols))
        w, wv = dev_rows(rng.standard_normal((E * rows, cols)) * cols ** -0.5, BF16, pad64(cols))
        out = torch.full((m, pad64(rows)), 7.0, dtype=torch.float32, device="cuda")
        L.check(lib.lbk_dense_linear(ctx.handle, compute, x.data_ptr(), x.shape[1], m, w.data_ptr(), w.shape[1], w.shape[0], cols, 0, rows, 0,
                                     out.data_ptr(), out.shape[1], 1, offs.data_ptr(), E, _st()))
        got, lo = out.cpu().numpy(), 0
        for e, c in enumerate(counts):
            want = xv[lo:lo + c] @ wv[e * rows:(e + 1) * rows].T
            if c:
                assert np.abs(got[lo:lo + c, :rows] - want).max() < 2e-5 * max(1.0, np.abs(want).max())
            lo += c
        assert (got[:, rows:] == 7.0).all()
    ctx.check_device_error()


# heads, kv_heads, dim, vdim, window, keep_first, scale, bias
ATTN = [(8, 2, 64, 64, 40, 5, 0.125, 1), (6, 1, 96, 48, 130, 20, 0.1, 1), (4, 4, 32, 128, 1, 0, 0.3, 1), (5, 5, 40, 24, 64, 200, 0.2, 1),
        (24, 1, 128, 128, 128, 1, 0.09, 1), (40, 2, 16, 16, 200, 130, 0.25, 1), (3, 1, 160, 192, 70, 9, 0.08, 1), (2, 1, 300, 272, 33, 2, 0.06, 1),
        (8, 8, 128, 64, 0, 0, 0.09, 0), (16, 4, 80, 112, 0, 0, 0.1, 1), (7, 7, 56, 8, 129, 128, 0.13, 1)]


def make_attention(rng, case, b, cap, compute):
    import torch
    H, G, dim, vdim = case[:4]
    dp, vp = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    dt = torch.bfloat16 if compute == BF16 else torch.float32
    k = torch.zeros(b, G, cap, dp, dtype=dt)
    v = torch.zeros(b, G, cap, vp, dtype=dt)
    k[..., :dim] = torch.from_numpy(rng.standard_normal((b, G, cap, dim))).to(dt)
    v[..., :vdim] = torch.from_numpy(rng.standard_normal((b, G, cap, vdim))).to(dt)
    return k, v, dp, vp, dt


def edge_keys(i, window, keep):
    """Keys just inside and just outside what position i sees, and the first and last kept ones."""
    out = [0, keep - 1, keep, i]
    if window:
        out += [i - window + 1, i - window]
    return sorted({j for j in out if 0 <= j <= i})


def spike(k, q_row, scale, dim, j):
    """Key j becomes a copy of the query that scores about 60 above the others: seeing it or not decides the row."""
    import torch
    d = q_row / torch.linalg.vector_norm(q_row.float()).to(q_row.dtype) ** 2
    k[j, :dim] = (60.0 / scale * d.float()).to(k.dtype)


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("case", ATTN)
def test_attention_rows(ctx, po, compute, case):
    """Rows of a prompt or a portion (from position 0, from the middle, of one or two rows), random keys, then keys
    that stand out at every edge of one row's view in turn: just inside and just outside the window, the last kept
    token and the first that is not."""
    import torch
    L, lib = _lib()
    H, G, dim, vdim, window, keep, scale, bias = case
    rng = np.random.default_rng(H * 1000 + dim)
    b, cap, seq = 2, 420, 1
    mask = {"size": window or 1 << 30, "keep_first": keep}
    for pos0, n in ((0, 1), (0, 300), (0, 130), (131, 2), (127, 7), (250, 150), (399, 9), (200, 64)):
        k, v, dp, vp, dt = make_attention(rng, case, b, cap, compute)
        k[:, :, pos0 + n:] = float("nan")          # what lies past the written positions must not matter
        v[:, :, pos0 + n:] = float("nan")
        q = torch.zeros(n, H, dp, dtype=dt)
        q[..., :dim] = torch.from_numpy(rng.standard_normal((n, H, dim))).to(dt)
        row = int(rng.integers(0, n))
        i = pos0 + row
        for spiked in [None] + edge_keys(i, window, keep):
            k2 = k.clone()
            if spiked is not None:
                for g in range(G):
                    spike(k2[seq, g], q[row, g * (H // G), :dim], scale, dim, spiked)
            qd, kd, vd = q.cuda(), k2.cuda(), v.cuda()
            pitch = pad64(H * vdim)
            out = torch.zeros(n, pitch, dtype=dt, device="cuda")
            pos = torch.tensor([pos0], dtype=torch.int32, device="cuda")
            L.check(lib.lbk_attn_window(ctx.handle, compute, qd.data_ptr(), kd.data_ptr(), vd.data_ptr(), pos.data_ptr(), n, seq, H, G, dim, dp,
                                        vdim, vp, cap, scale, window, keep, bias, None, out.data_ptr(), pitch, _st()))
            total = pos0 + n
            kf, vf = k2[seq, :, :total, :dim].double().numpy(), v[seq, :, :total, :vdim].double().numpy()
            rows = range(n) if spiked is None else [row]
            qf = q[list(rows), :, :dim].double().numpy()
            want = reference(po, qf, kf, vf, scale, mask, [pos0 + r for r in rows], bias)
            got = out.float().cpu().numpy()[list(rows), :H * vdim].reshape(len(list(rows)), H, vdim)
            tol = 2e-5 if compute == F32 else 1.2e-2
            assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (pos0, n, row, spiked)
    ctx.check_device_error()


def reference(po, q, k, v, scale, mask, qpos, bias):
    """po.attention with or without the bias; k, v [G, n, d]."""
    kt, vt = k.transpose(1, 0, 2), v.transpose(1, 0, 2)
    if bias:
        return po.attention(q, kt, vt, scale, mask, qpos, np.arange(kt.shape[0]))
    see = po.visible(qpos, np.arange(kt.shape[0]), mask)
    out = np.empty((q.shape[0], q.shape[1], vt.shape[2]))
    for h in range(q.shape[1]):
        g = h // (q.shape[1] // kt.shape[1])
        s = np.where(see, q[:, h] @ kt[:, g].T * scale, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = p / p.sum(-1, keepdims=True) @ vt[:, g]
    return out


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("case", ATTN)
def test_attention_decode(ctx, po, compute, case):
    """One new token for each of several sequences at positions around every edge, the keys at the edges standing out
    in turn; a large batch (fewer slices) and a long cache (many slices)."""
    import torch
    L, lib = _lib()
    H, G, dim, vdim, window, keep, scale, bias = case
    rng = np.random.default_rng(H * 77 + dim)
    mask = {"size": window or 1 << 30, "keep_first": keep}
    edge = (window or 64) + keep
    for b, cap, posv in ((1, 900, [899]), (5, 420, [0, min(419, edge), min(419, edge - 1), 63, 417]), (16, 300, list(range(3, 300, 19))[:16])):
        k, v, dp, vp, dt = make_attention(rng, case, b, cap, compute)
        for s, p in enumerate(posv):
            k[s, :, p + 1:] = float("nan")
            v[s, :, p + 1:] = float("nan")
        q = torch.zeros(b, H, dp, dtype=dt)
        q[..., :dim] = torch.from_numpy(rng.standard_normal((b, H, dim))).to(dt)
        for which in range(-1, 6):
            k2 = k.clone()
            if which >= 0:
                for s, p in enumerate(posv):
                    e = edge_keys(p, window, keep)
                    for g in range(G):
                        spike(k2[s, g], q[s, g * (H // G), :dim], scale, dim, e[which % len(e)])
            scratch = torch.empty(int(lib.lbk_attn_window_scratch(b, H, vp)), device="cuda")
            qd, kd, vd = q.cuda(), k2.cuda(), v.cuda()
            pitch = pad64(H * vdim)
            out = torch.zeros(b, pitch, dtype=dt, device="cuda")
            pos = torch.tensor(posv, dtype=torch.int32, device="cuda")
            L.check(lib.lbk_attn_window(ctx.handle, compute, qd.data_ptr(), kd.data_ptr(), vd.data_ptr(), pos.data_ptr(), b, -1, H, G, dim, dp,
                                        vdim, vp, cap, scale, window, keep, bias, scratch.data_ptr(), out.data_ptr(), pitch, _st()))
            got = out.float().cpu().numpy()[:, :H * vdim].reshape(b, H, vdim)
            for s, p in enumerate(posv):
                want = reference(po, q[s:s + 1, :, :dim].double().numpy(), k2[s, :, :p + 1, :dim].double().numpy(),
                                 v[s, :, :p + 1, :vdim].double().numpy(), scale, mask, [p], bias)[0]
                tol = 2e-5 if compute == F32 else 1.2e-2
                assert np.abs(got[s] - want).max() < tol * max(1.0, np.abs(want).max()), (b, p, which)
    ctx.check_device_error()


@pytest.mark.parametrize("n,E,top", [(1, 3, 1), (5, 16, 16), (100, 7, 2), (257, 300, 6), (40, 1000, 32)])
def test_route(ctx, po, n, E, top):
    """The chosen experts, their scores (of a softmax over all experts, not renormalised), and the sorted order: every
    (token, choice) has its own sorted row inside its expert's range, holding the token's values."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(n)
    z = (3.0 * rng.standard_normal((n, E + 1))).astype(np.float32)
    z[0, :E] = 1.0                                  # equal scores: the lower index first
    x = torch.from_numpy(rng.standard_normal((n, 128))).to(torch.bfloat16).cuda()
    zd = torch.from_numpy(z).cuda()
    i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device="cuda")
    ids, place, offs, wts = i32(n, top), i32(n, top), i32(E + 1), torch.zeros(n, top, device="cuda")
    xs = torch.zeros(n * top, 128, dtype=torch.bfloat16, device="cuda")
    scratch = torch.full((int(lib.lbk_moe_route_ints(n, E, top)),), 12345, dtype=torch.int32, device="cuda")
    L.check(lib.lbk_moe_route(ctx.handle, zd.data_ptr(), E + 1, n, E, top, scratch.data_ptr(), x.data_ptr(), 128, xs.data_ptr(), ids.data_ptr(),
                              wts.data_ptr(), place.data_ptr(), offs.data_ptr(), _st()))
    want_ids, want_w = po.route(z[:, :E].astype(np.float64), np.eye(E), top)
    assert np.array_equal(ids.cpu().numpy(), want_ids)
    assert np.abs(wts.cpu().numpy() - want_w).max() < 1e-6
    counts = np.bincount(want_ids.reshape(-1), minlength=E)
    o = offs.cpu().numpy()
    assert o[0] == 0 and np.array_equal(np.diff(o), counts)
    pl = place.cpu().numpy()
    assert sorted(pl.reshape(-1).tolist()) == list(range(n * top))
    assert (pl >= o[want_ids]).all() and (pl < o[want_ids + 1]).all()
    for k in range(top):
        assert torch.equal(xs[torch.from_numpy(pl[:, k]).long().cuda()], x)
    ctx.check_device_error()


def test_argument_errors(ctx):
    """Shapes the kernels do not take are refused with a message, before any launch."""
    import torch
    L, lib = _lib()
    x = torch.zeros(2, 64, dtype=torch.bfloat16, device="cuda")
    with pytest.raises(L.LbkError, match="pitches"):
        L.check(lib.lbk_dense_linear(ctx.handle, BF16, x.data_ptr(), 64, 2, x.data_ptr(), 60, 2, 60, 0, 2, 0, x.data_ptr(), 64, 0, None, 0, _st()))
    with pytest.raises(L.LbkError, match="has 2 rows for 2"):
        L.check(lib.lbk_dense_linear(ctx.handle, BF16, x.data_ptr(), 64, 2, x.data_ptr(), 64, 2, 64, 1, 2, 0, x.data_ptr(), 64, 0, None, 0, _st()))
    pos = torch.zeros(1, dtype=torch.int32, device="cuda")
    with pytest.raises(L.LbkError, match="inconsistent"):
        L.check(lib.lbk_attn_window(ctx.handle, BF16, x.data_ptr(), x.data_ptr(), x.data_ptr(), pos.data_ptr(), 1, 0, 3, 2, 16, 16, 16, 16, 4, 1.0, 0, 0,
                                    1, None, x.data_ptr(), 64, _st()))
    with pytest.raises(L.LbkError, match="at most 512"):
        L.check(lib.lbk_attn_window(ctx.handle, BF16, x.data_ptr(), x.data_ptr(), x.data_ptr(), pos.data_ptr(), 1, 0, 1, 1, 520, 528, 16, 16, 4, 1.0, 0, 0,
                                    1, None, x.data_ptr(), 64, _st()))
    with pytest.raises(L.LbkError, match="routing"):
        L.check(lib.lbk_moe_route(ctx.handle, x.data_ptr(), 4, 1, 4, 5, x.data_ptr(), None, 64, None, None, None, None, None, _st()))
