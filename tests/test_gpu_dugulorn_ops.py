"""The mechanisms of the Dugulorn family one by one (RMS sandwich norm, biased and silu projections, rotation and latent
cache rows, latent attention in both forms, both recurrences, gated norm) against the plain numpy functions of its oracle,
in both compute types, at sizes that are not multiples of anything."""
import ctypes as C

import numpy as np
import pytest

pytestmark = pytest.mark.gpu
BF16, F32 = 0, 1


@pytest.fixture(scope="module")
def do():
    from oracle import dugulorn_oracle
    return dugulorn_oracle


def _lib():
    from lemonade_burn_b200 import _lib as L
    return L, L.load()


def _st():
    import torch
    return torch.cuda.current_stream().cuda_stream


def pad(n, k=64):
    return (n + k - 1) // k * k


def typed(compute):
    import torch
    return torch.bfloat16 if compute == BF16 else torch.float32


def rows(a, compute, pitch=None, dtype=None):
    """numpy [m, n] -> (device rows of the compute type with zeros up to `pitch`, exact values)."""
    import torch
    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).to(dtype or typed(compute))
    out = torch.zeros(a.shape[0], pitch or a.shape[1], dtype=t.dtype)
    out[:, :a.shape[1]] = t
    return out.cuda(), t.double().numpy()


def cuda(a, dtype=None):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype or torch.float32).cuda()


def ints(*v):
    import torch
    return torch.tensor(v, dtype=torch.int32, device="cuda")


@pytest.mark.parametrize("n", [4, 66, 250, 1000, 2560, 8190, 9001])
def test_rms_sandwich_norm(ctx, do, n):
    """x += norm(y) * w_post, then the sum itself or its norm: rows with a mean far from zero (taking it off would show)."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(n)
    for m, with_y, with_w in ((1, True, False), (5, True, True), (3, False, True)):
        x, y = (rng.standard_normal((m, n)) + 3.0).astype(np.float32), (2.0 * rng.standard_normal((m, n)) - 20.0).astype(np.float32)
        wp, w, eps = rng.standard_normal(n).astype(np.float32), rng.standard_normal(n).astype(np.float32), 1e-2
        xd, yd, wpd, wd, of = cuda(x), cuda(y), cuda(wp), cuda(w), torch.zeros(m, n, device="cuda")
        oe = torch.zeros(m, pad(n), dtype=torch.bfloat16, device="cuda")
        L.check(lib.lbk_sandwich_rms_norm(ctx.handle, xd.data_ptr(), yd.data_ptr() if with_y else None, wpd.data_ptr() if with_y else None,
                                          wd.data_ptr() if with_w else None, m, n, eps, of.data_ptr(), oe.data_ptr(), pad(n), _st()))
        wx = x.astype(np.float64) + (do.rms_norm(y.astype(np.float64), wp, eps) if with_y else 0.0)
        want = do.rms_norm(wx, w, eps) if with_w else wx
        assert np.abs(xd.cpu().numpy() - wx).max() < 2e-5 * np.abs(wx).max()
        assert np.abs(of.cpu().numpy() - want).max() < 3e-5 * np.abs(want).max()
        assert np.abs(oe.float().cpu().numpy()[:, :n] - want).max() < 2.0 ** -8 * np.abs(want).max() and not oe[:, n:].any()
    ctx.check_device_error()


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("r,c", [(40, 72), (130, 200), (97, 40), (700, 512)])
def test_projection_with_bias_and_activation(ctx, do, compute, r, c):
    """A bias on every output row; squared relu; silu on the front rows only; at token counts of every kernel."""
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(r)
    for m in (1, 2, 8, 9, 17, 130, 300):
        x, xv = rows(rng.standard_normal((m, c)), compute, pad(c))
        w, wv = rows(rng.standard_normal((r, c)) * c ** -0.5, BF16, pad(c))
        b = rng.standard_normal(r).astype(np.float32)
        bd = cuda(b)
        for bias, act, act_rows, f32 in ((True, 0, r, 1), (True, 1, r, 0), (False, 2, r - 11, 0), (True, 2, r, 0)):
            out = torch.full((m, pad(r)), 7.0, dtype=torch.float32 if f32 else typed(compute), device="cuda")
            L.check(lib.lbk_dense_linear_act(ctx.handle, compute, x.data_ptr(), x.shape[1], m, w.data_ptr(), w.shape[1], r, c, bd.data_ptr() if bias else None, act, act_rows,
                                             out.data_ptr(), pad(r), f32, _st()))
            want = xv @ wv.T + (b if bias else 0.0)
            if act and not f32:
                want[:, :act_rows] = (do.relu2 if act == 1 else do.silu)(want[:, :act_rows])
            got = out.float().cpu().numpy()
            tol = 1e-5 if out.dtype == torch.float32 else 2.0 ** -8
            assert np.abs(got[:, :r] - want).max() <= tol * max(1.0, np.abs(want).max()), (m, bias, act)
            assert (got[:, r:] == 7.0).all()
    ctx.check_device_error()


def test_rotation_frequencies(do):
    """Plain and YaRN-scaled: the ramp inside, at and beyond both ends of the pairs, one pair, equal ends."""
    from lemonade_burn_b200 import mixers
    for dims, base, yarn in ((2, 100.0, None), (64, 1e4, None), (64, 1e4, (4.0, 4096, 32.0, 1.0)), (10, 500.0, (2.0, 64, 8.0, 2.0)), (32, 1e6, (16.0, 100000, 40.0, 0.5)),
                             (6, 10.0, (3.0, 7, 1.0, 1.0)), (128, 1e4, (8.0, 20, 1.0, 0.25))):
        f, m = mixers.rotation_frequencies(dims, base, yarn)
        sc = None if yarn is None else dict(zip(("factor", "original", "fast", "slow"), yarn))
        wf, wm = do.frequencies({"dims": dims, "base": base, "scaling": sc})
        assert np.allclose(f, wf, rtol=1e-13) and abs(m - wm) < 1e-6


# heads, dim, rot_dim, vdim, kv_rank, q_rank, base, yarn
LATENT = [(4, 16, 8, 16, 16, 24, 100.0, None), (3, 24, 10, 40, 56, 33, 5e3, (2.0, 64, 8.0, 1.0)), (20, 32, 16, 48, 128, 80, 1e4, None),
          (40, 64, 32, 64, 200, 96, 1e4, (4.0, 128, 32.0, 1.0)), (17, 128, 64, 128, 500, 72, 1e6, None), (1, 40, 2, 17, 70, 5, 10.0, None),
          (33, 48, 128, 200, 512, 40, 1e4, None)]


class Latent:
    """A random layer of `case`: descriptor, weights, and a cache filled by lbk_latent_prep."""

    def __init__(self, ctx, do, case, compute, b, cap, seed=0):
        from lemonade_burn_b200 import mixers
        import torch
        self.L, self.lib = _lib()
        self.ctx, self.do, self.compute, self.b, self.cap = ctx, do, compute, b, cap
        H, dim, rot, vd, kr, qr, base, yarn = case
        self.H, self.dim, self.rot, self.vd, self.kr, self.qr = H, dim, rot, vd, kr, qr
        self.rotation = {"dims": rot, "base": base, "scaling": None if yarn is None else dict(zip(("factor", "original", "fast", "slow"), yarn))}
        f, m = mixers.rotation_frequencies(rot, base, yarn)
        self.freq = torch.from_numpy(f).cuda()
        self.d = mixers.LatentDesc(H, dim, rot, vd, kr, qr, self.freq.data_ptr(), m)
        ref = C.byref(self.d)
        self.pitch, self.key_at = self.lib.lbk_latent_pitch(ref), self.lib.lbk_latent_key_at(ref)
        self.qp, self.rot_at = self.lib.lbk_latent_query_pitch(ref), self.lib.lbk_latent_query_rot_at(ref)
        self.rng = np.random.default_rng(seed + H)
        self.cache = torch.zeros(b, cap, self.pitch, dtype=typed(compute), device="cuda")
        self.ukv, self.ukv_v = rows(self.rng.standard_normal((H * (dim + vd), kr)) * kr ** -0.5, BF16, pad(kr))
        self.q_norm, self.kv_norm = (1.0 + 0.2 * self.rng.standard_normal(n) for n in (qr, kr))
        self.scale = float((dim + rot) ** -0.5)

    def prep(self, z, seq, pos, own=True, eps=1e-3):
        import torch
        n = z.shape[0]
        zd = cuda(z)
        qn, kn = cuda(self.q_norm), cuda(self.kv_norm)
        cq = torch.zeros(n, pad(self.qr), dtype=typed(self.compute), device="cuda")
        p = ints(*pos)
        self.L.check(self.lib.lbk_latent_prep(self.ctx.handle, self.compute, C.byref(self.d), zd.data_ptr(), z.shape[1], n, seq, p.data_ptr(), self.cap, qn.data_ptr(),
                                              kn.data_ptr(), eps, cq.data_ptr(), pad(self.qr), self.cache.data_ptr() if own else None, _st()))
        torch.cuda.synchronize()
        return cq

    def want_rows(self, z, positions, eps=1e-3):
        z = z.astype(np.float32).astype(np.float64)
        kv = z[:, self.qr:self.qr + self.kr + self.rot]
        n32 = lambda a: a.astype(np.float32).astype(np.float64)
        return (self.do.rms_norm(z[:, :self.qr], n32(self.q_norm), eps), self.do.rms_norm(kv[:, :self.kr], n32(self.kv_norm), eps),
                self.do.rotate(kv[:, self.kr:], positions, self.rotation))

    def fill(self, seq, n):
        """Random cache rows 0 .. n - 1 of a sequence, everything behind them poison."""
        import torch
        self.cache[seq, :n] = 0
        self.cache[seq, :n, :self.kr] = cuda(self.rng.standard_normal((n, self.kr)), self.cache.dtype)
        self.cache[seq, :n, self.key_at:self.key_at + self.rot] = cuda(self.rng.standard_normal((n, self.rot)), self.cache.dtype)
        self.cache[seq, n:] = float("nan")
        torch.cuda.synchronize()

    def latents(self, seq, n):
        c = self.cache[seq, :n].double().cpu().numpy()
        return c[:, :self.kr], c[:, self.key_at:self.key_at + self.rot]

    def queries(self, n):
        import torch
        q = torch.zeros(n, self.H, self.qp, dtype=typed(self.compute))
        q[..., :self.dim] = torch.from_numpy(self.rng.standard_normal((n, self.H, self.dim))).to(q.dtype)
        q[..., self.rot_at:self.rot_at + self.rot] = torch.from_numpy(self.rng.standard_normal((n, self.H, self.rot))).to(q.dtype)
        return q

    def attend(self, q, seq, pos, gate, length=0):
        import torch
        n = q.shape[0]
        qd, gd, p = q.cuda(), cuda(gate), ints(*pos)
        out = torch.full((n, pad(self.H * self.vd)), 7.0, dtype=typed(self.compute), device="cuda")
        work = torch.full((int(self.lib.lbk_latent_work_bytes(self.ctx.handle, self.compute, C.byref(self.d), n, self.cap, length)),), 255, dtype=torch.uint8, device="cuda")
        self.L.check(self.lib.lbk_latent_attn(self.ctx.handle, self.compute, C.byref(self.d), qd.data_ptr(), n, seq, p.data_ptr(), self.cap, self.cache.data_ptr(),
                                              self.ukv.data_ptr(), pad(self.kr), self.scale, gd.data_ptr(), self.H, length, work.data_ptr(), out.data_ptr(), out.shape[1], _st()))
        self.ctx.check_device_error()
        got = out.float().cpu().numpy()
        assert (got[:, self.H * self.vd:] == 7.0).all()
        return got[:, :self.H * self.vd].reshape(n, self.H, self.vd)

    def want(self, q, seq, pos, gate, n_keys):
        """One row's output from keys and values written out head by head."""
        c, kr = self.latents(seq, n_keys)
        qf = q.double().numpy()
        qr = self.do.rotate(qf[None, :, self.rot_at:self.rot_at + self.rot], [pos], self.rotation)[0]
        out = np.empty((self.H, self.vd))
        for h in range(self.H):
            k = c @ self.ukv_v[h * self.dim:(h + 1) * self.dim].T
            v = c @ self.ukv_v[self.H * self.dim + h * self.vd:self.H * self.dim + (h + 1) * self.vd].T
            s = (k @ qf[h, :self.dim] + kr @ qr[h]) * self.scale
            e = np.exp(s - s.max())
            out[h] = e / e.sum() @ v * self.do.sigmoid(np.float64(np.float32(gate[h])))
        return out


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("case", LATENT)
def test_latent_prep(ctx, do, case, compute):
    """Normed query latents, and cache rows of a portion and of one token per sequence, at small and very large positions
    (angles of many thousand turns); other rows and the padding stay; a layer without a latent writes nothing."""
    t = Latent(ctx, do, case, compute, 3, 70000 if case[0] == 4 else 300)
    tol = 2e-6 if compute == F32 else 2.0 ** -8
    for seq, pos, n in ((1, [5], 7), (-1, [0, t.cap - 1, 77], 3)):
        t.cache.fill_(0)
        z = t.rng.standard_normal((n, t.qr + t.kr + t.rot + t.H)) * 3.0 + 1.0
        cq = t.prep(z, seq, pos)
        where = [(seq, pos[0] + i) for i in range(n)] if seq >= 0 else list(enumerate(pos))
        wq, wc, wr = t.want_rows(z, [p for _, p in where])
        got = t.cache.double().cpu().numpy()
        assert np.abs(cq.double().cpu().numpy()[:, :t.qr] - wq).max() < tol * np.abs(wq).max()
        for i, (s, p) in enumerate(where):
            row = got[s, p]
            assert np.abs(row[:t.kr] - wc[i]).max() < tol * np.abs(wc[i]).max()
            assert np.abs(row[t.key_at:t.key_at + t.rot] - wr[i]).max() < 2 * tol * np.abs(wr[i]).max()
            assert not row[t.kr:t.key_at].any() and not row[t.key_at + t.rot:].any()
            got[s, p] = 0
        assert not got.any()
        before = t.cache.clone()
        cq2 = t.prep(np.concatenate([z[:, :t.qr], z[:, t.qr + t.kr + t.rot:]], 1), seq, pos, own=False)
        assert (t.cache == before).all() and (cq2 == cq).all()
    ctx.check_device_error()


def far_key(t, q, seq, pos, key):
    """The cache row `key` becomes one whose score of head 0 stands about 40 above the others'."""
    import torch
    u = t.do.rotate(q[None, 0, t.rot_at:t.rot_at + t.rot].double().numpy(), [pos], t.rotation)[0]
    t.cache[seq, key, t.key_at:t.key_at + t.rot] = cuda(u / (u @ u) * 40.0 / t.scale, t.cache.dtype)
    torch.cuda.synchronize()


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("case", LATENT)
def test_latent_attention_of_single_tokens(ctx, do, case, compute):
    """One token per sequence at positions around the 64-position chunks and slices, poison behind them; then a key that
    decides the row at the first, an edge and the last position. A token sees exactly the positions up to its own."""
    b, cap = 6, 700
    t = Latent(ctx, do, case, compute, b, cap)
    pos = [0, 63, 64, 127, 350, 699]
    for s, p in enumerate(pos):
        t.fill(s, p + 1)
    q, gate = t.queries(b), t.rng.standard_normal((b, t.H))
    tol = 3e-5 if compute == F32 else 1.5e-2
    for edge in (None, lambda p: 0, lambda p: p, lambda p: p // 64 * 64, lambda p: max(0, p - 64)):
        if edge:
            for s, p in enumerate(pos):
                far_key(t, q[s], s, p, edge(p))
        got = t.attend(q, -1, pos, gate)
        for s, p in enumerate(pos):
            want = t.want(q[s], s, p, gate[s], p + 1)
            assert np.abs(got[s] - want).max() < tol * max(0.3, np.abs(want).max()), (s, p)
    ctx.check_device_error()


@pytest.mark.parametrize("compute,expand", [(BF16, False), (BF16, True), (F32, False)])
@pytest.mark.parametrize("case", LATENT)
def test_latent_attention_of_rows(ctx, do, case, compute, expand):
    """Rows of a portion in both forms: from position 0, from the middle, single rows, more than a tile; keys that decide
    a row just before it and at its own position, none of them visible to the row in front."""
    t = Latent(ctx, do, case, compute, 2, 420)
    if expand and not t.lib.lbk_latent_expand_supported(C.byref(t.d)):
        assert case[1] > 128 or case[3] > 128 or pad(case[1]) + pad(case[2]) > 192
        return
    tol = 3e-5 if compute == F32 else 1.5e-2
    for p0, n in ((0, 1), (0, 150), (131, 2), (127, 40), (290, 129)):
        t.fill(1, p0 + n)
        q, gate = t.queries(n), t.rng.standard_normal((n, t.H))
        mid = n // 2
        far_key(t, q[mid], 1, p0 + mid, p0 + mid)
        if n > 2:
            far_key(t, q[-1], 1, p0 + n - 1, p0 + n - 2)
        got = t.attend(q, 1, [p0], gate, p0 + n if expand else 0)
        for i in sorted({0, mid, max(0, mid - 1), max(0, n - 2), n - 1}):
            want = t.want(q[i], 1, p0 + i, gate[i], p0 + i + 1)
            assert np.abs(got[i] - want).max() < tol * max(0.3, np.abs(want).max()), (p0, n, i)
    ctx.check_device_error()


# heads, kv_heads, dim, vdim, taps
RECUR = [(3, 3, 24, 40, 4), (6, 2, 48, 17, 3), (1, 1, 64, 64, 1), (4, 2, 128, 96, 4), (5, 1, 33, 130, 2), (2, 2, 200, 24, 7), (2, 1, 256, 300, 4)]


class Recur:
    """A random layer of `case` with states and convolution inputs of `b` sequences."""

    def __init__(self, ctx, do, case, compute, delta, b=1, seed=0, strong=False):
        from lemonade_burn_b200 import mixers
        import torch
        self.L, self.lib = _lib()
        self.ctx, self.do, self.compute, self.delta = ctx, do, compute, delta
        H, G, d, vd, taps = case
        G = G if delta else H
        self.H, self.G, self.d, self.vd, self.taps, self.b = H, G, d, vd, taps, b
        self.desc = mixers.RecurrenceDesc(int(delta), H, G, d, vd, taps)
        self.rng = np.random.default_rng(seed + H + d)
        self.ch = 2 * G * d + H * vd
        self.pitch = pad(self.ch)
        self.state = torch.full((b * int(self.lib.lbk_recurrence_state_floats(C.byref(self.desc))),), float("nan"), device="cuda")  # a state at position 0 is not read
        self.ring = torch.full((b, taps, self.ch), float("nan"), dtype=typed(compute), device="cuda")
        self.rr = 24
        self.records = torch.full((int(self.lib.lbk_recurrence_record_floats(C.byref(self.desc), self.rr)),), float("nan"), device="cuda")
        self.decay = np.linspace(0.3, 1.0, H).astype(np.float32)
        self.conv = (self.rng.standard_normal((self.ch, taps)) * 0.7).astype(np.float32)
        self.a_log = (self.rng.standard_normal(H) * (1.0 if strong else 0.5) + (2.0 if strong else 0.0)).astype(np.float32)
        self.bias = (self.rng.standard_normal(H * d) + (3.0 if strong else -1.0)).astype(np.float32)
        self.dev = [cuda(x) for x in (self.decay, np.ascontiguousarray(self.conv.T), self.a_log, self.bias)]

    def inputs(self, n):
        """(x, a, b) of n tokens, as exact values."""
        _, x = rows(self.rng.standard_normal((n, self.ch)), self.compute)
        return x, self.rng.standard_normal((n, self.H * self.d)).astype(np.float32), self.rng.standard_normal((n, self.H)).astype(np.float32)

    def run(self, tok, seq, pos, active=None, cap=1000):
        import torch
        x, a, b = tok
        xd, _ = rows(x, self.compute, self.pitch)
        ad, bd, p = cuda(a), cuda(b), ints(*pos)
        act = ints(*active) if active is not None else None
        o = torch.full((len(x), self.H * self.vd), 7.0, device="cuda")
        dec, conv, al, dt = self.dev
        self.L.check(self.lib.lbk_recurrence(self.ctx.handle, self.compute, C.byref(self.desc), xd.data_ptr(), self.pitch, len(x), seq, p.data_ptr(),
                                             act.data_ptr() if act is not None else None, cap, dec.data_ptr(), conv.data_ptr(), self.ring.data_ptr(), ad.data_ptr(), al.data_ptr(),
                                             dt.data_ptr(), bd.data_ptr(), self.state.data_ptr(), self.records.data_ptr(), self.rr, o.data_ptr(), _st()))
        self.ctx.check_device_error()
        return o.cpu().numpy().reshape(len(x), self.H, self.vd)

    def want(self, tok):
        """o of a whole sequence, token by token."""
        x, a, b = (np.asarray(v, dtype=np.float64) for v in tok)
        n, H, G, d, vd, do = len(x), self.H, self.G, self.d, self.vd, self.do
        k0, v0 = G * d, 2 * G * d
        if not self.delta:
            return do.lightning_core(x[:, :k0].reshape(n, H, d), x[:, k0:v0].reshape(n, H, d), x[:, v0:].reshape(n, H, vd), self.decay.astype(np.float64))
        y = do.silu(do.short_conv(x, self.conv.astype(np.float64)))
        of = np.arange(H) // (H // G)
        q = (do.unit(y[:, :k0].reshape(n, G, d)) * d ** -0.5)[:, of]
        k = do.unit(y[:, k0:v0].reshape(n, G, d))[:, of]
        g = np.exp(-np.exp(self.a_log.astype(np.float64))[:, None] * do.softplus(a + self.bias).reshape(n, H, d))
        return do.delta_core(q, k, y[:, v0:].reshape(n, H, vd), g, do.sigmoid(b))


def cut(tok, lo, hi):
    return tuple(v[lo:hi] for v in tok)


def agree(got, want, compute):
    # the inputs are exact in both types; bf16 only has the faster silu of the convolution
    assert np.abs(got - want).max() < 2e-5 * max(1.0, np.abs(want).max()), (np.abs(got - want).max(), np.abs(want).max())


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("delta", [False, True])
@pytest.mark.parametrize("case", RECUR)
def test_recurrence_rows_and_single_tokens(ctx, do, case, delta, compute):
    """A sequence in one piece (several runs of records, a ragged last one), in portions down to one and two tokens, and
    token by token; portions and single tokens taking turns. The state and ring of another sequence stay."""
    n = 61
    t = Recur(ctx, do, case, compute, delta, b=2)
    tok = t.inputs(n)
    want = t.want(tok)
    for cuts in ([n], [1] * n, [2] * 30 + [1], [3, 8, 1, 1, 7, 16, 2, 9, 14], [8, 24, 29], [25, 36]):
        for one in (False, True):                      # single tokens as a row of the sequence, or as a step of the batch
            other = t.state[:len(t.state) // 2].clone(), t.ring[0].clone()
            at, got = 0, []
            for c in cuts:
                piece = cut(tok, at, at + c)
                if one and c == 1:
                    both = tuple(np.concatenate([v, v]) for v in piece)
                    got.append(t.run(both, -1, [0, at], active=[0, 1])[1:])
                else:
                    got.append(t.run(piece, 1, [at]))
                at += c
            agree(np.concatenate(got), want, compute)
            now = t.state[:len(t.state) // 2], t.ring[0]
            assert all((a.nan_to_num(123.0) == b.nan_to_num(123.0)).all() for a, b in zip(other, now))
            if 1 not in cuts:
                break


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("delta", [False, True])
@pytest.mark.parametrize("case", RECUR)
def test_recurrence_of_a_batch(ctx, do, case, delta, compute):
    """Sequences of unequal lengths advance together, one not taking part now and then; one starts again at position 0 in
    the place of another (its state and ring are not cleared in between)."""
    t = Recur(ctx, do, case, compute, delta, b=3)
    toks = [t.inputs(40) for _ in range(3)]
    want = [t.want(k) for k in toks]
    at = [0, 5, 17]
    for s in range(3):
        if at[s]:
            agree(t.run(cut(toks[s], 0, at[s]), s, [0]), want[s][:at[s]], compute)
    for step in range(12):
        active = [1, int(step % 3 != 1), 1]
        x = tuple(np.concatenate([toks[s][i][at[s]:at[s] + 1] for s in range(3)]) for i in range(3))
        got = t.run(x, -1, at, active=active)
        for s in range(3):
            if active[s]:
                agree(got[s], want[s][at[s]], compute)
                at[s] += 1
        if step == 6:
            toks[2], at[2] = t.inputs(40), 0
            want[2] = t.want(toks[2])


@pytest.mark.parametrize("delta", [False, True])
def test_long_and_strongly_decaying_recurrences(ctx, do, delta):
    """1500 tokens (an error that grows would show), and decays so strong that products of a few of them are zero."""
    t = Recur(ctx, do, (2, 1, 64, 40, 4), F32, delta)
    tok = t.inputs(1500)
    want = t.want(tok)
    got = t.run(tok, 0, [0], cap=1500)
    assert np.abs(got - want).max() < 4e-5 * np.abs(want).max()
    t = Recur(ctx, do, (2, 2, 40, 24, 3), F32, delta, strong=True)
    t.decay[:] = [1e-12, 1.0]
    t.dev[0] = cuda(t.decay)
    tok = t.inputs(50)
    agree(np.concatenate([t.run(cut(tok, 0, 27), 0, [0]), t.run(cut(tok, 27, 50), 0, [27])]), t.want(tok), F32)


@pytest.mark.parametrize("taps", [2, 4, 5])
def test_every_tap_reaches_back_across_a_cut(ctx, do, taps):
    """A convolution whose only weight is on its oldest input: each token's vectors are those of the token taps - 1 before
    it, in the prompt, over a cut and in single steps."""
    t = Recur(ctx, do, (2, 2, 16, 16, taps), F32, True)
    t.conv[:] = 0.0
    t.conv[:, 0] = 1.0
    t.dev[1] = cuda(np.ascontiguousarray(t.conv.T))
    tok = t.inputs(30)
    want = t.want(tok)
    for cuts in ([30], [10, 1, 1, 2, 1, 15], [1] * 30, [2, 3, 2, 23]):
        at, got = 0, []
        for c in cuts:
            got.append(t.run(cut(tok, at, at + c), -1 if c == 1 else 0, [at]))
            at += c
        agree(np.concatenate(got), want, F32)


@pytest.mark.parametrize("compute", [BF16, F32])
@pytest.mark.parametrize("m,n,group", [(1, 40, 40), (3, 120, 24), (5, 17, 1), (2, 2560, 2560), (7, 600, 300), (2, 4096, 128)])
def test_gated_norm(ctx, do, compute, m, n, group):
    import torch
    L, lib = _lib()
    rng = np.random.default_rng(n)
    o, w = (rng.standard_normal((m, n)) * 5.0 + 2.0).astype(np.float32), rng.standard_normal(group).astype(np.float32)
    g, gv = rows(rng.standard_normal((m, n)), compute, pad(n))
    od, wd, out = cuda(o), cuda(w), torch.full((m, pad(n)), 7.0, dtype=typed(compute), device="cuda")
    L.check(lib.lbk_gated_norm(ctx.handle, compute, od.data_ptr(), m, n, group, wd.data_ptr(), g.data_ptr(), pad(n), 0.03, out.data_ptr(), pad(n), _st()))
    want = (do.rms_norm(o.astype(np.float64).reshape(m, -1, group), w, 0.03)).reshape(m, n) * do.sigmoid(gv)
    got = out.double().cpu().numpy()
    assert np.abs(got[:, :n] - want).max() < (2e-6 if compute == F32 else 2.0 ** -8) * np.abs(want).max() and (got[:, n:] == 7.0).all()


def test_refused_arguments(ctx):
    """Shapes the kernels do not take are refused with a message, before any launch."""
    import torch
    from lemonade_burn_b200 import mixers
    L, lib = _lib()
    x = torch.zeros(4096, device="cuda")
    p = x.data_ptr()
    with pytest.raises(L.LbkError, match="activation"):
        L.check(lib.lbk_dense_linear_act(ctx.handle, F32, p, 64, 1, p, 64, 2, 60, None, 9, 2, p, 64, 0, _st()))
    with pytest.raises(L.LbkError, match="ragged groups"):
        L.check(lib.lbk_gated_norm(ctx.handle, F32, p, 1, 10, 3, p, p, 64, 1e-5, p, 64, _st()))
    d = mixers.LatentDesc(2, 16, 3, 16, 16, 16, p, 1.0)
    with pytest.raises(L.LbkError, match="odd"):
        L.check(lib.lbk_latent_prep(ctx.handle, F32, C.byref(d), p, 64, 1, 0, p, 4, p, p, 1e-5, p, 64, p, _st()))
    d = mixers.LatentDesc(2, 16, 4, 16, 600, 16, p, 1.0)
    with pytest.raises(L.LbkError, match="at most 512"):
        L.check(lib.lbk_latent_attn(ctx.handle, BF16, C.byref(d), p, 1, 0, p, 4, p, p, 640, 1.0, p, 2, 0, p, p, 64, _st()))
    r = mixers.RecurrenceDesc(0, 1, 1, 300, 16, 1)
    with pytest.raises(L.LbkError, match="at most 256"):
        L.check(lib.lbk_recurrence(ctx.handle, F32, C.byref(r), p, 1024, 1, 0, p, None, 4, p, None, None, None, None, None, None, p, p, 8, p, _st()))
