"""Layered decoders on the GPU against the plain oracle: each kernel alone, then whole models in both number formats."""
import numpy as np
import pytest

from fusekit_b200 import _native as N
from fusekit_b200 import checkpoint as CK
from fusekit_b200 import task_graph as TG
from fusekit_b200.model_spec import LAYERED_CONFIGS, LoopSpec
from fusekit_b200.runtime import attach
from oracle import layered as OL
from tests import layered_models as LM

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 3e-5, 0.05


def up(v, m):
    return (v + m - 1) // m * m


class Dev:
    """Device buffers of one test, freed together."""

    def __init__(self, rt):
        self.rt, self.ptrs = rt, []

    def put(self, a):
        p = self.rt.to_device(np.ascontiguousarray(a)); self.ptrs.append(p)
        return p

    def new(self, nbytes):
        p = self.rt.alloc(nbytes); self.ptrs.append(p)
        return p

    def act(self, a, f32, ld=None):
        """Rows as activations, zero-padded to ld columns."""
        a = np.asarray(a, np.float32)
        if ld is not None and ld != a.shape[-1]:
            a = np.concatenate([a, np.zeros(a.shape[:-1] + (ld - a.shape[-1],), np.float32)], -1)
        return self.put(a if f32 else LM.bits(a))

    def get(self, p, shape, f32):
        return self.rt.download(p, shape, np.float32) if f32 else LM.values(self.rt.download(p, shape, np.uint16))

    def close(self):
        for p in self.ptrs:
            N.check(self.rt.L.fk_free(self.rt.h, p), "fk_free")


@pytest.fixture
def dev(runtime):
    d = Dev(runtime)
    yield d
    d.close()


def rows_weight(rt, w_bits):
    n, k = w_bits.shape
    kp = up(k, 64)
    wid = rt.weight_alloc(n, kp, 16)
    rt.weight_upload_rows(wid, 0, np.concatenate([w_bits, np.zeros((n, kp - k), np.uint16)], 1))
    rt.weight_keep_rows(wid)
    return wid


def close(got, want, tol, what=""):
    err = np.abs(got - want).max() / max(1e-30, np.abs(want).max())
    assert err <= tol, f"{what}: {err:.3g} > {tol}"


# ------------------------------------------------------------------ kernels alone
# row counts around the 64- and 128-row tiles, outputs around the 64 / 128 / 256-column tiles, K below and above one stage; the
# last two are large enough for the widest tiles and for several tiles per block
@pytest.mark.parametrize("m,n,k", [(2, 3, 8), (64, 64, 64), (65, 129, 200), (129, 40, 600), (300, 257, 72), (2050, 2300, 136), (4100, 1536, 328)])
@pytest.mark.parametrize("f32", [0, 1])
def test_linear_rows(runtime, dev, m, n, k, f32):
    if f32 and m > 2000:
        m = 260
    rng = np.random.default_rng(m + n + k)
    x, w = LM.rounded(rng.standard_normal((m, k))), LM.bits(rng.standard_normal((n + 5, k)))
    wid, ldx, ldy = rows_weight(runtime, w), up(k, 64), up(n, 8)
    xd, y, yf = dev.act(x, f32, ldx), dev.new(m * ldy * 4), dev.new(m * n * 4)
    runtime.state_set(0, 0)
    runtime.launch(N.Task.make(N.TASK_LINEAR_ROWS, -1, {0: xd, 1: wid, 2: y}, [m, 0, n, ldx, ldy, f32, N.ACT_RELU_SQUARED, 0]))
    runtime.launch(N.Task.make(N.TASK_LINEAR_ROWS, -1, {0: xd, 1: wid, 2: yf}, [m, 5, n, ldx, n, f32, 256, 0]))       # from row 5, fp32 out
    assert runtime.state_get()[2] == 0
    z = x.astype(np.float64) @ LM.values(w).T
    close(dev.get(y, (m, ldy), f32)[:, :n], np.maximum(z[:, :n], 0) ** 2, 2e-6 if f32 else 5e-3, "relu squared")
    close(dev.get(yf, (m, n), 1), z[:, 5:], 2e-6, "fp32 output")


@pytest.mark.parametrize("counts", [[0, 130, 0, 1, 64, 0], [5, 0, 0], [1] * 40, [0, 0, 300, 129, 128, 127, 1]])
@pytest.mark.parametrize("f32", [0, 1])
def test_grouped_linear_rows_with_empty_experts(runtime, dev, counts, f32):
    rng = np.random.default_rng(len(counts))
    E, n, k, m = len(counts), 72, 104, sum(counts)
    x, w = LM.rounded(rng.standard_normal((m, k))), LM.bits(rng.standard_normal((E * n, k)))
    off = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
    ldx, ldy = up(k, 64), up(n, 64)
    y = dev.new(m * ldy * 4)
    runtime.state_set(0, 0)
    runtime.launch(N.Task.make(N.TASK_LINEAR_ROWS, -1, {0: dev.act(x, f32, ldx), 1: rows_weight(runtime, w), 2: y, 3: dev.put(off)}, [m, 0, n, ldx, ldy, f32, 0, E]))
    assert runtime.state_get()[2] == 0
    wv = LM.values(w).reshape(E, n, k).astype(np.float64)
    want = np.concatenate([x[off[e]:off[e + 1]] @ wv[e].T for e in range(E)])
    close(dev.get(y, (m, ldy), f32)[:, :n], want, 2e-6 if f32 else 5e-3)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("d", [40, 333, 2048])
def test_residual_norm_rows(runtime, dev, d, f32):
    rng = np.random.default_rng(d)
    M, top, eps, ld = 5, 3, 1e-3, up(d, 64)
    x, add = rng.standard_normal((M, d)).astype(np.float32), rng.standard_normal((M, d)).astype(np.float32)
    y, ye = LM.rounded(rng.standard_normal((M, d))), LM.rounded(rng.standard_normal((M * top, d)))
    post, w = LM.rounded(1 + 0.2 * rng.standard_normal(d)), LM.rounded(1 + 0.2 * rng.standard_normal(d))
    slot, wt = rng.permutation(M * top).astype(np.int32), rng.random((M, top)).astype(np.float32)
    xd, h = dev.put(x), dev.new(M * ld * 4)
    yd, yed, pd, wd = dev.act(y, f32, ld), dev.act(ye, f32, ld), dev.put(LM.bits(post)), dev.put(LM.bits(w))
    # everything at once, in place
    runtime.launch(N.Task.make(N.TASK_RESIDUAL_NORM_ROWS, 0, {0: xd, 1: yd, 2: pd, 3: dev.put(add), 4: xd, 5: wd, 6: h, 8: yed, 9: dev.put(slot), 10: dev.put(wt)},
                               [d, M, f32, ld, top, ld], [eps]))
    yy = y.astype(np.float64) + (ye[slot].reshape(M, top, d) * wt[:, :, None]).sum(1)
    xn = x + OL.rms_norm(yy, post, eps) + add
    close(dev.get(xd, (M, d), 1), xn, 2e-6, "x")
    close(dev.get(h, (M, ld), f32)[:, :d], OL.rms_norm(xn, w, eps), 2e-6 if f32 else 5e-3, "h")
    # two chosen rows, x left alone
    runtime.launch(N.Task.make(N.TASK_RESIDUAL_NORM_ROWS, 0, {0: xd, 5: wd, 6: h, 7: dev.put(np.array([3, 1], np.uint32))}, [d, 2, f32, ld, 0, ld], [eps]))
    close(dev.get(h, (M, ld), f32)[:2, :d], OL.rms_norm(xn[[3, 1]], w, eps), 2e-6 if f32 else 5e-3, "chosen rows")


def attention_case(rng, H, G, dim, vdim, maps, n, far):
    """Unit-scale heads; with ``far`` the last query and the key at position ``far`` point the same way in every head and map, so
    that this one score stands out by a wide margin (and its value row is large)."""
    q, k, v = rng.standard_normal((n, H, maps, dim)), rng.standard_normal((n, G, maps, dim)), rng.standard_normal((n, G, vdim))
    if far is not None:
        u = rng.standard_normal(dim); u *= np.sqrt(dim) / np.linalg.norm(u)
        q[-1] = u; k[far] = u
        v[far] *= 5
    return q, k, v


def oracle_heads(q, k, v, m, lam, diff, eps, gate, pos0):
    """Attention of the query rows (already normalised) at positions pos0 ..: [T, H * vdim]."""
    T, H = q.shape[:2]
    G, dv = k.shape[1], v.shape[2]
    out = np.zeros((T, H, dv))
    for h in range(H):
        g = h // (H // G)
        a = [OL.softmax_attention(q[:, h, j], k[:, g, j], v[:, g], m, pos0) for j in range(q.shape[2])]
        out[:, h] = OL.differential_combine(a[0], a[1], lam, diff, eps) if len(a) == 2 else a[0]
        out[:, h] *= OL.sigmoid(gate[:, h:h + 1])
    return out.reshape(T, -1)


ATT = [(4, 2, 24, 40, 2), (2, 1, 64, 128, 2), (3, 3, 8, 8, 2), (5, 1, 40, 72, 1), (10, 1, 128, 64, 2), (2, 2, 130, 200, 2), (2, 1, 72, 256, 2), (1, 1, 16, 300, 1), (4, 4, 33, 21, 2)]


@pytest.mark.parametrize("H,G,dim,vdim,maps", ATT)
@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("before,rows", [(0, 2), (0, 65), (61, 5), (70, 64), (127, 70), (640, 2)])
def test_store_and_attention_rows(runtime, dev, H, G, dim, vdim, maps, f32, before, rows):
    """The q/k norm, the cache store and the attention of ``rows`` positions after ``before`` cached ones; a far key that only the
    last position's query matches, at the start, around 64-key tile edges and just inside the portion."""
    rng = np.random.default_rng(H * 1000 + dim + before)
    n, cap, eps, scale, lam, diff = before + rows, before + rows + 3, 1e-4, 1.1 * dim ** -0.5, 0.6, 0.35
    dp, vp, ld, ldo = up(dim, 8), up(vdim, 8), up((H + G) * maps * dim + G * vdim + H, 64), up(H * vdim, 64)
    sz, tol = 4 if f32 else 2, 3e-5 if f32 else 2e-2
    for far in sorted({0, min(63, n - 1), min(64, n - 1), before, n - 1}):
        q, k, v = attention_case(rng, H, G, dim, vdim, maps, n, far)
        q, k, v = LM.rounded(q[before:]).astype(np.float64), LM.rounded(k).astype(np.float64), LM.rounded(v).astype(np.float64)
        gate = LM.rounded(rng.standard_normal((rows, H)))
        qn, kn = LM.rounded(1 + 0.2 * rng.standard_normal(dim)), LM.rounded(1 + 0.2 * rng.standard_normal(dim))
        kk, qq = OL.rms_norm(k, kn, eps), OL.rms_norm(q, qn, eps)
        ck, cv = np.zeros((G * maps, cap, dp), np.float32), np.zeros((G, cap, vp), np.float32)
        ck[:, :before, :dim] = kk[:before].transpose(1, 2, 0, 3).reshape(G * maps, before, dim)
        cv[:, :before, :vdim] = v[:before].transpose(1, 0, 2)
        raw = np.concatenate([q.reshape(rows, -1), k[before:].reshape(rows, -1), v[before:].reshape(rows, -1), gate], 1)
        rawd, ckd, cvd = dev.act(raw, f32, ld), dev.act(ck, f32), dev.act(cv, f32)
        qd, out = dev.new(rows * H * maps * dp * sz), dev.new(rows * ldo * sz)
        runtime.state_set(0, before)
        runtime.launch(N.Task.make(N.TASK_QK_NORM_STORE_ROWS, 0, {0: rawd, 1: dev.put(LM.bits(qn)), 2: dev.put(LM.bits(kn)), 3: qd, 4: ckd, 5: cvd},
                                   [H, G, dim, vdim, cap, rows, f32 | maps << 8, ld], [eps]))
        gp = rawd + (ld and ((H + G) * maps * dim + G * vdim)) * sz
        runtime.launch(N.Task.make(N.TASK_ATTENTION_ROWS, 0, {0: qd, 1: ckd, 2: cvd, 3: out, 4: gp}, [H, G, dim, vdim, cap, rows, f32 | maps << 8, ld],
                                   [scale, lam, diff, eps]))
        assert runtime.state_get()[2] == 0
        kc = dev.get(ckd, (G * maps, cap, dp), f32)
        close(kc[:, before:n, :dim], kk[before:].transpose(1, 2, 0, 3).reshape(G * maps, rows, dim), 2e-6 if f32 else 5e-3, "stored keys")
        assert not kc[:, n:].any()
        want = oracle_heads(qq, kk, v, scale, lam, diff, eps, gate, before)
        got = dev.get(out, (rows, ldo), f32)[:, :H * vdim]
        close(got, want, tol, f"far key {far}")
        close(got[-1], want[-1], tol, f"last position, far key {far}")


@pytest.mark.parametrize("H,G,dim,vdim,maps", ATT)
@pytest.mark.parametrize("f32", [0, 1])
def test_attention_decode(runtime, dev, H, G, dim, vdim, maps, f32):
    """One position with the keys split over 1, 3 and many blocks; far keys at the first key, around 32-key and split edges."""
    rng = np.random.default_rng(H + dim)
    eps, scale, lam, diff = 1e-4, 1.1 * dim ** -0.5, 0.6, 0.35
    dp, vp, tiles, sz = up(dim, 8), up(vdim, 8), -(-(H // G * maps) // 8), 4 if f32 else 2
    for pos, splits in ((0, 1), (0, 5), (31, 1), (32, 3), (300, 3), (1000, 20)):
        n, cap = pos + 1, pos + 9
        per = up(-(-n // splits), 32)
        for far in sorted({0, min(per - 1, pos), min(per, pos), pos}):
            q, k, v = attention_case(rng, H, G, dim, vdim, maps, n, far)
            k, v = LM.rounded(k).astype(np.float64), LM.rounded(v).astype(np.float64)
            q, gate = q[-1:].astype(np.float32).astype(np.float64), rng.standard_normal((1, H)).astype(np.float32)
            qn, kn = LM.rounded(1 + 0.2 * rng.standard_normal(dim)), LM.rounded(1 + 0.2 * rng.standard_normal(dim))
            kk = OL.rms_norm(k, kn, eps)
            ck, cv = np.zeros((G * maps, cap, dp), np.float32), np.zeros((G, cap, vp), np.float32)
            ck[:, :pos, :dim] = kk[:pos].transpose(1, 2, 0, 3).reshape(G * maps, pos, dim)
            cv[:, :pos, :vdim] = v[:pos].transpose(1, 0, 2)
            raw = np.concatenate([q.reshape(-1), k[-1].reshape(-1), v[-1].reshape(-1), gate[0]]).astype(np.float32)
            ckd, cvd, out = dev.act(ck, f32), dev.act(cv, f32), dev.new(H * vdim * 4)
            part, cnt = dev.new(G * tiles * splits * 8 * (vp + 2) * 4), dev.new(G * tiles * 4)
            runtime.state_set(0, pos)
            t = N.Task.make(N.TASK_ATTENTION_DECODE, 0, {0: dev.put(raw), 1: dev.put(LM.bits(qn)), 2: dev.put(LM.bits(kn)), 3: ckd, 4: cvd, 5: out, 6: part, 7: cnt},
                            [H, G, dim, vdim, cap, 1, f32 | maps << 8, splits], [scale, lam, diff, eps])
            want = oracle_heads(OL.rms_norm(q, qn, eps), kk, v, scale, lam, diff, eps, gate, pos)[0]
            for again in range(2):                       # the split counters are left as they were found
                runtime.launch(t)
                assert runtime.state_get()[2] == 0
                close(runtime.download(out, (H * vdim,), np.float32), want, 3e-5 if f32 else 1e-2, f"pos {pos}, {splits} splits, far {far}")
            vc = dev.get(cvd, (G, cap, vp), f32)
            assert np.array_equal(vc[:, pos, :vdim], v[-1].astype(np.float32)) and not vc[:, n:].any()


def test_positions_outside_the_cache_are_reported(runtime, dev):
    runtime.state_set(0, 4)
    buf = dev.new(1 << 16)
    runtime.launch(N.Task.make(N.TASK_ATTENTION_DECODE, 0, {i: buf for i in range(8)}, [1, 1, 8, 8, 4, 0, 1 | 256, 1], [1.0, 0.0, 0.0, 1e-6]))
    assert runtime.state_get()[2] & 0x100000
    runtime.state_set(0, 0)


@pytest.mark.parametrize("k,n,pend", [(8, 5, 1), (100, 300, 0), (1000, 77, 1), (2048, 3001, 1), (4500, 16, 1)])
def test_norm_linear(runtime, dev, k, n, pend):
    rng = np.random.default_rng(k)
    eps, row0 = 1e-3, n // 3
    x, y, add = (rng.standard_normal(k).astype(np.float32) for _ in range(3))
    post, w = LM.rounded(1 + 0.2 * rng.standard_normal(k)), LM.rounded(1 + 0.2 * rng.standard_normal(k))
    W = LM.bits(rng.standard_normal((n, k)))
    wid, out, xo, ho = rows_weight(runtime, W), dev.new(n * 4), dev.new(k * 4), dev.new(k * 4)
    bufs = {0: dev.put(x), 5: dev.put(LM.bits(w)), 6: wid, 7: out, 8: ho}
    if pend:
        bufs.update({1: dev.put(y), 2: dev.put(LM.bits(post)), 3: dev.put(add), 4: xo})
    runtime.launch(N.Task.make(N.TASK_NORM_LINEAR, 0, bufs, [k, n, N.ACT_RELU_SQUARED, row0], [eps]))
    xn = x + OL.rms_norm(y.astype(np.float64), post, eps) + add if pend else x.astype(np.float64)
    h = OL.rms_norm(xn, w, eps)
    z = LM.values(W).astype(np.float64) @ h
    z[row0:] = np.maximum(z[row0:], 0) ** 2
    close(runtime.download(ho, (k,), np.float32), h, 2e-6, "h")
    close(runtime.download(out, (n,), np.float32), z, 3e-6, "y")
    if pend:
        close(runtime.download(xo, (k,), np.float32), xn, 2e-6, "x")
    # plain product, and the greedy choice with ties going to the lowest index
    W2 = W.copy(); W2[n - 1] = W2[n // 2] = W2[int(np.argmax(LM.values(W).astype(np.float64) @ x))]
    runtime.state_set(0, 7)
    runtime.launch(N.Task.make(N.TASK_NORM_LINEAR, 0, {0: bufs[0], 6: rows_weight(runtime, W2), 7: out, 9: dev.new(8192), 10: dev.new(4)}, [k, n, 0, 0], [eps]))
    z = LM.values(W2).astype(np.float64) @ x
    close(runtime.download(out, (n,), np.float32), z, 3e-6, "plain")
    tok, off, err = runtime.state_get()
    assert (off, err) == (8, 0) and tok == int(np.flatnonzero(z == z.max())[0])


@pytest.mark.parametrize("E,top,ff,ffs,D", [(1, 1, 8, 0, 16), (7, 3, 40, 56, 88), (70, 6, 300, 20, 130), (33, 33, 16, 520, 64), (1000, 64, 24, 8, 72)])
def test_moe_decode(runtime, dev, E, top, ff, ffs, D):
    rng = np.random.default_rng(E)
    h, z = rng.standard_normal(D).astype(np.float32), rng.standard_normal(E).astype(np.float32)
    if E > 2:
        z[E // 2] = z[E // 2 - 1]                        # equal logits: the lower index first
    up_, down = LM.bits(rng.standard_normal((E * ff, D)) * D ** -0.5), LM.bits(rng.standard_normal((E * D, ff)) * ff ** -0.5)
    act, sel, wt, y, sa = dev.new(top * ff * 4), dev.new(top * 4), dev.new(top * 4), dev.new(D * 4), rng.random(max(ffs, 1)).astype(np.float32)
    runtime.launch(N.Task.make(N.TASK_MOE_UP, 0, {0: dev.put(z), 1: dev.put(h), 2: rows_weight(runtime, up_), 3: act, 4: sel, 5: wt}, [D, E, top, ff, N.ACT_RELU_SQUARED]))
    idx, w = OL.route(z.astype(np.float64)[None], top)
    assert runtime.download(sel, (top,), np.int32).tolist() == idx[0].tolist()
    close(runtime.download(wt, (top,), np.float32), w[0], 2e-6)
    b = {0: act, 1: sel, 2: wt, 3: rows_weight(runtime, down), 6: y}
    want = 0.0
    if ffs:
        sd = LM.bits(rng.standard_normal((D, ffs)) * ffs ** -0.5)
        b.update({4: dev.put(sa[:ffs]), 5: rows_weight(runtime, sd)})
        want = LM.values(sd).astype(np.float64) @ sa[:ffs]
    runtime.launch(N.Task.make(N.TASK_MOE_DOWN, 0, b, [D, E, top, ff, ffs]))
    U, Dn = LM.values(up_).reshape(E, ff, D).astype(np.float64), LM.values(down).reshape(E, D, ff).astype(np.float64)
    for j, e in enumerate(idx[0]):
        want = want + w[0, j] * OL.expert(U[e], Dn[e], h.astype(np.float64))
    close(runtime.download(y, (D,), np.float32), want, 3e-6)


@pytest.mark.parametrize("rows,E,top", [(2, 3, 1), (37, 70, 6), (300, 9, 9), (129, 300, 4)])
@pytest.mark.parametrize("f32", [0, 1])
def test_moe_route_rows(runtime, dev, rows, E, top, f32):
    rng = np.random.default_rng(rows)
    D, ldl = 72, up(E, 64)
    ld = up(D, 64)
    z, h = rng.standard_normal((rows, ldl)).astype(np.float32), LM.rounded(rng.standard_normal((rows, D)))
    z[:, 1 % E] = z[:, 0]
    S = rows * top
    b = {0: dev.put(z), 1: dev.act(h, f32, ld), 2: dev.new(S * 4), 3: dev.new(S * 4), 4: dev.new(S * 4), 5: dev.new(E * 4), 6: dev.new(S * 4), 7: dev.new((E + 1) * 4),
         8: dev.new(S * ld * 4)}
    for _ in range(2):                                   # the counts start from zero every time
        runtime.launch(N.Task.make(N.TASK_MOE_ROUTE_ROWS, 0, b, [rows, E, top, ldl, ld, f32]))
    idx, w = OL.route(z[:, :E].astype(np.float64), top)
    sel, slot = runtime.download(b[3], (rows, top), np.int32), runtime.download(b[6], (rows, top), np.int32)
    off = runtime.download(b[7], (E + 1,), np.int32)
    assert np.array_equal(sel, idx)
    close(runtime.download(b[2], (rows, top), np.float32), w, 2e-6)
    assert np.array_equal(np.diff(off), np.bincount(idx.ravel(), minlength=E)) and off[0] == 0
    assert sorted(slot.ravel()) == list(range(S))
    assert ((slot >= off[idx]) & (slot < off[idx + 1])).all()
    got = dev.get(b[8], (S, ld), f32)
    assert np.array_equal(got[slot.ravel(), :D], np.repeat(h, top, 0)) and not got[:, D:].any()


# ------------------------------------------------------------------ whole models
def check_logits(got, want, dtype, what=""):
    e = LM.logit_error(got, want)
    if dtype == "float32":
        assert e.max() <= F32_TOL, f"{what}: {e.max():.3g}"
    else:                                                # a close router call may fall the other way at a position
        assert np.median(e) <= BF16_TOL and (e > 3 * BF16_TOL).mean() <= 0.08, f"{what}: median {np.median(e):.3g}, worst {e.max():.3g}"


PORTIONS = {"whole": None, "twos": [2], "mixed": [7, 2, 33, 1, 64, 3], "single": [1]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(LM.SPECS))
def test_portions_of_a_prompt_match_the_oracle(runtime, name, dtype):
    """Logits at every position, whatever the portions; slots are reused between the sequences, and two are open at once."""
    s = LM.SPECS[name]
    t = LM.random_tensors(s, 5)
    toks = np.random.default_rng(2).integers(0, s.vocab, 150)
    want = LM.oracle(s, t).forward(toks)
    e = LM.engine(s, t, 170, dtype, runtime=runtime, max_rows=100)
    other, slots = e.open_sequence(), set()
    other.append(toks[::-1][:20])
    results = {}
    for how, sizes in PORTIONS.items():
        seq, got, p, j = e.open_sequence(), [], 0, 0
        slots.add(seq.slot)
        while p < len(toks):
            n = len(toks) if sizes is None else min(sizes[j % len(sizes)], len(toks) - p)
            got.append(seq.append(toks[p:p + n], list(range(n)))); p += n; j += 1
        seq.close()
        results[how] = np.concatenate(got)
        check_logits(results[how], want, dtype, f"{name} {how}")
    assert len(slots) == 1 and other.slot not in slots
    # the sequence that stayed open goes on undisturbed
    o2 = LM.oracle(s, t)
    w2 = o2.forward(toks[::-1][:25])
    check_logits(other.append(toks[::-1][20:25], [0, 1, 2, 3, 4]), w2[20:], dtype, "kept sequence")
    other.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_decides_the_output(runtime, dtype):
    """One layer whose keys and queries single out the position of a marker token: the logits after a late query token must follow
    the value stored hundreds of positions earlier, through prompts, portions and decoding."""
    s = LM.spec([LM.LayerSpec(LM.A(2, 1, 16, 24, 1.5, 0.3), None)], hidden=64, vocab=50)
    t = LM.random_tensors(s, 9)
    emb = LM.values(t["embed"]).copy()
    emb[:, 0] = 0.0; emb[:, 1] = 0.0
    emb[7, 0] = 12.0; emb[8, 1] = 12.0                   # 7: marker (keys), 8: asks for it (queries)
    t["embed"] = LM.bits(emb)
    q, k = LM.values(t["l0.mix.q"]).copy(), LM.values(t["l0.mix.k"]).copy()
    u = np.random.default_rng(0).standard_normal(16)
    q[:, 1] = np.tile(u, 4) * 3; k[:, 0] = np.tile(u, 2) * 3
    t["l0.mix.q"], t["l0.mix.k"] = LM.bits(q), LM.bits(k)
    n = 700
    e = LM.engine(s, t, n + 4, dtype, runtime=runtime)
    for far in (0, 1, 63, 64, 511, n - 2):
        toks = np.random.default_rng(far).integers(10, s.vocab, n); toks[far] = 7; toks[-1] = 8
        without = toks.copy(); without[far] = 11
        want, blind = (LM.oracle(s, t).forward(x)[-1:] for x in (toks, without))
        assert LM.logit_error(blind, want)[0] > 0.2      # the key matters
        for cut in (0, n - 1, n - 2, 64):
            seq = e.open_sequence()
            if cut:
                seq.append(toks[:cut])
            got = seq.append(toks[cut:], [n - cut - 1])
            seq.close()
            assert LM.logit_error(got, want)[0] < (F32_TOL if dtype == "float32" else BF16_TOL), (far, cut)


def test_long_decoding_stays_on_the_oracle(runtime):
    s = LM.spec([LM.LayerSpec(LM.A(2, 1, 8, 16, 0.5, 0.3), LM.M(4, 2, 16, 8))], hidden=32, vocab=60, loop=LoopSpec(0, 1, 2))
    t = LM.random_tensors(s, 4)
    toks = np.random.default_rng(3).integers(0, s.vocab, 400)
    want = LM.oracle(s, t).forward(toks)
    e = LM.engine(s, t, 400, "float32", runtime=runtime)
    seq = e.open_sequence()
    seq.append(toks[:2])
    got = np.concatenate([seq.append(toks[i:i + 1], [0]) for i in range(2, 400)])
    check_logits(got, want[2:], "float32")
    seq.close()


@pytest.mark.parametrize("name", ["mixed", "many-rows"])
def test_greedy_and_sampled_generation(runtime, tmp_path, name):
    """From a model directory through the framework's loader and entry points: the device's greedy chain equals the oracle's, a
    second request in the same slot too, and top-k 1 sampling is greedy."""
    s = LM.SPECS[name]
    t = LM.random_tensors(s, 8)
    LM.write_model(tmp_path / "m", s, t)
    e, ck = CK.load_engine(str(tmp_path / "m"), 120, dtype="float32", runtime=runtime)
    try:
        for seed, n in ((0, 40), (1, 1), (2, 3)):
            prompt = np.random.default_rng(seed).integers(0, s.vocab, n).tolist()
            o, want, toks = LM.oracle(s, t), [], prompt
            for _ in range(30):
                z = o.forward(toks)[-1]
                toks = [int(np.argmax(z))]; want += toks
            assert e.complete(prompt, 30).tolist() == want
            assert e.complete(prompt, 5, temperature=0.7, top_k=1).tolist() == want[:5]
            a, b = (e.complete(prompt, 6, 1.2, top_k=8, seed=3).tolist() for _ in range(2))
            assert a == b and max(a) < s.vocab
    finally:
        ck.close()


@pytest.mark.parametrize("which", ["model", "layered", "older"])
def test_command_line(tmp_path, capsys, which):
    from fusekit_b200.generate import main
    if which == "model":
        s = LM.SPECS["mixed"]
        t = LM.random_tensors(s, 8)
        LM.write_model(tmp_path / "m", s, t)
        o, want, toks = LM.oracle(s, t), [], [3, 1, 4]
        for _ in range(6):
            toks = [int(np.argmax(o.forward(toks)[-1]))]; want += toks
        assert main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt", "3,1,4", "--max-tokens", "6"]) == 0
        assert [int(v) for v in capsys.readouterr().out.split(",")] == want
        return
    args = ["--config", "tiny-fatulix" if which == "layered" else "tiny-qwen", "--prompt", "3,1,4", "--max-tokens", "6"]
    assert main(args) == 0 and main(args + ["--temperature", "0.8", "--top-k", "1"]) == 0
    a, b = capsys.readouterr().out.split()
    assert a == b and len(a.split(",")) == 6


def test_registered_shape_through_attach(runtime):
    """The registry's small shape with synthetic weights: graph capture from the JSON text decodes the same tokens."""
    import json
    e = attach(LAYERED_CONFIGS["tiny-fatulix"], 64, runtime=runtime)
    e.load_synthetic()
    first = e.prefill([5, 9, 2, 44])
    a, _ = e.generate(first, 4, 20)
    e.prefill([5, 9, 2, 44])
    e.capture_json(json.dumps(e.task_graph()))
    b, _ = e.generate(first, 4, 20)
    assert a.tolist() == b.tolist() and len(set(a.tolist())) > 1
    assert TG.K_MOEUP in [t.kind for t in e.replay]


def test_bad_requests_are_refused_on_the_host(runtime):
    s = LM.SPECS["one-layer"]
    e = LM.engine(s, LM.random_tensors(s), 16, runtime=runtime)
    for call in (lambda: e.step([s.vocab], 0), lambda: e.step([], 0), lambda: e.step([1] * 17, 0), lambda: e.step([1], 16), lambda: e.step([1, 2], 0, [2]),
                 lambda: e.prefill([1, 2], 15), lambda: e.decode_chunk(10, 1, 7), lambda: e.release(e.free[0])):
        with pytest.raises(ValueError):
            call()
    with pytest.raises(ValueError):
        LM.engine(s, LM.random_tensors(s), 16, "float16", runtime=runtime)
    with pytest.raises(N.FusekitError):                  # a weight in the streaming layout is not rows
        wid = runtime.weight_alloc(16, 64, 16)
        runtime.weight_finalize(wid)
        runtime.launch(N.Task.make(N.TASK_NORM_LINEAR, 0, {0: 4096, 6: wid, 7: 4096}, [64, 16, 0, 0], [1e-6]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_writes_the_asked_logits(runtime, tmp_path, dtype):
    import json
    from fusekit_b200.trace import TraceRunner
    s = LM.SPECS["mixed"]
    t = LM.random_tensors(s, 6)
    LM.write_model(tmp_path / "m", s, t)
    e, ck = CK.load_engine(str(tmp_path / "m"), 64, dtype=dtype, runtime=runtime)
    toks = np.random.default_rng(1).integers(0, s.vocab, 30).tolist()
    want = LM.oracle(s, t).forward(toks)
    r = TraceRunner(e, str(tmp_path))
    assert r.step(json.loads(json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:20], "want": [3, 19]}], "end": []}))) == 0
    r.step({"step": 1, "entries": [{"id": "a", "tokens": toks[20:28], "want": []}], "end": []})
    r.step({"step": 2, "entries": [{"id": "a", "tokens": toks[28:], "want": [1]}], "end": ["a"]})
    r.step({"step": 3, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}], "end": ["b"]})
    assert not (tmp_path / "1.f32").exists() and not r.live and len(e.caches) == 1
    for step, rows in ((0, [3, 19]), (2, [29]), (3, [0])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), s.vocab)
        e_ = LM.logit_error(got, want[rows])
        assert e_.max() < (F32_TOL if dtype == "float32" else 4 * BF16_TOL)
    ck.close()
