"""Parallel blocks of the layered decoders on the GPU against the plain oracle: each kernel alone, then whole models in both number
formats."""
import numpy as np
import pytest

from fusekit_b200 import _native as N
from fusekit_b200 import checkpoint as CK
from fusekit_b200 import task_graph as TG
from fusekit_b200.layered import rotation_table
from fusekit_b200.model_spec import LAYERED_CONFIGS
from fusekit_b200.runtime import attach
from oracle import layered as OL
from tests import layered_models as LM
from tests.test_gpu_layered import BF16_TOL, F32_TOL, check_logits, close, dev, rows_weight, up  # noqa: F401  (dev is a fixture)

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("d", [40, 333, 1200, 2048, 5120])
def test_block_norm_rows(runtime, dev, d, f32):
    """Two normed and one plain pending output, and the cases with fewer; layer norm of rows with a large common offset, and RMS norm."""
    rng = np.random.default_rng(d)
    M, eps, ld = 5, 1e-3, up(d, 64)
    x = (rng.standard_normal((M, d)) + 20).astype(np.float32)
    y = [LM.rounded(rng.standard_normal((M, d)) * 3) for _ in range(3)]
    post, w, b = (LM.rounded(1 + 0.3 * rng.standard_normal(n)) for n in ((3, d), d, d))
    yd = [dev.act(v, f32, ld) for v in y]
    wd, bd, pd = dev.put(LM.bits(w)), dev.put(LM.bits(b)), dev.put(LM.bits(post))
    h = dev.new(M * ld * 4)
    for np_, nn, bias in ((0, 0, 1), (1, 0, 1), (1, 1, 0), (2, 0, 1), (2, 2, 1), (3, 2, 1), (3, 3, 0)):
        xd = dev.put(x)
        bufs = {0: xd, 4: xd, 5: wd, 6: h, 8: bd if bias else 0, 9: pd, **{1 + j: yd[j] for j in range(np_)}}
        runtime.launch(N.Task.make(N.TASK_BLOCK_NORM_ROWS, 0, bufs, [d, M, f32, ld, ld, np_, nn], [eps, 0.5]))
        xn = x.astype(np.float64)
        for j in range(np_):
            xn = xn + (0.5 * OL.rms_norm(y[j].astype(np.float64), post[j], eps) if j < nn else y[j])
        want = OL.layer_norm(xn, w, b, eps) if bias else OL.rms_norm(xn, w, eps)
        close(dev.get(xd, (M, d), 1), xn, 1e-6, "x")
        close(dev.get(h, (M, ld), f32)[:, :d], want, 1e-5 if f32 else 5e-3, f"h {np_} {nn}")
    runtime.launch(N.Task.make(N.TASK_BLOCK_NORM_ROWS, 0, {0: xd, 5: wd, 6: h, 7: dev.put(np.array([3, 1], np.uint32)), 8: bd}, [d, 2, f32, ld, ld, 0, 0], [eps, 0.5]))
    close(dev.get(h, (M, ld), f32)[:2, :d], OL.layer_norm(xn[[3, 1]], w, b, eps), 1e-5 if f32 else 5e-3, "chosen rows")
    close(dev.get(xd, (M, d), 1), xn, 1e-6, "x is left alone")


def block_columns(rng, k, silu, plain, exact, pairs):
    return LM.bits(rng.standard_normal((exact + 2 * pairs, k)) * 2 * k ** -0.5)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("m,k,silu,plain,exact,pairs", [(2, 40, 0, 32, 64, 3), (130, 72, 50, 96, 96, 70), (65, 200, 64, 64, 96, 0), (300, 136, 300, 320, 352, 333), (2050, 64, 1000, 1024, 1056, 700)])
def test_block_linear_rows(runtime, dev, m, k, silu, plain, exact, pairs, f32):
    rng = np.random.default_rng(m)
    if f32:
        m = min(m, 140)
    W, x, n, limit = block_columns(rng, k, silu, plain, exact, pairs), LM.rounded(rng.standard_normal((m, k))), exact + 2 * pairs, 0.9
    ldx, ldy, ld3 = up(k, 64), up(plain, 64), up(max(pairs, 1), 64)
    y, z, ff = dev.new(m * ldy * 4), dev.new(m * max(exact - plain, 1) * 4), dev.new(m * ld3 * 4)
    runtime.state_set(0, 0)
    runtime.launch(N.Task.make(N.TASK_BLOCK_LINEAR_ROWS, 0, {0: dev.act(x, f32, ldx), 1: rows_weight(runtime, W), 2: y, 3: z if exact > plain else 0, 4: ff if pairs else 0},
                               [m, plain, exact, n, ldy, ld3, f32, silu], [limit]))
    assert runtime.state_get()[2] == 0
    want = x.astype(np.float64) @ LM.values(W).T
    tol = 3e-6 if f32 else 5e-3
    got = dev.get(y, (m, ldy), f32)
    if silu:
        close(got[:, :silu], OL.silu(want[:, :silu]), tol, "silu")
    if plain > silu:
        close(got[:, silu:plain], want[:, silu:plain], tol, "plain")
    if exact > plain:
        close(dev.get(z, (m, exact - plain), 1), want[:, plain:exact], 3e-6, "fp32 columns")
    if pairs:
        got = dev.get(ff, (m, ld3), f32)
        close(got[:, :pairs], OL.clamped_glu(want[:, exact::2], want[:, exact + 1::2], limit), tol, "pairs")
        assert not got[:, pairs:].any()


# (H, G, dim, vdim, rotated dims): one head to a tile of rows and past it, sizes off every tile, above what the tensor-core form takes
ATT = [(4, 2, 24, 40, 16), (6, 3, 18, 22, 18), (3, 3, 64, 64, 0), (10, 1, 40, 72, 40), (2, 1, 128, 128, 128), (12, 1, 136, 200, 100), (1, 1, 8, 8, 2)]


def turned(u, pos, freqs):
    """The vector that rotation at ``pos`` takes to ``u``."""
    return OL.rotate_pairs(np.asarray(u, np.float64)[None, None], [-pos], freqs)[0, 0]


class AttentionCase:
    """Cached keys and values of n positions; the query at each position of ``asks`` and the key at ``far`` point the same way after
    rotation in every head, and the value there is large: whether that key is seen decides the output."""

    def __init__(self, rng, H, G, dim, vdim, rot, n, asks, far, window, keep):
        self.H, self.G, self.dim, self.vdim, self.window, self.keep, self.eps = H, G, dim, vdim, window, keep, 1e-4
        self.rot = LM.RotarySpec(rot, 50.0, LM.FrequencyScaling(4.0, 1.0, 3.0, 60.0))
        f = np.array(self.rot.frequencies())
        q, k, v = rng.standard_normal((n, H, dim)), rng.standard_normal((n, G, dim)), rng.standard_normal((n, G, vdim))
        u = rng.standard_normal(dim); u *= np.sqrt(dim) / np.linalg.norm(u)
        for p in asks:
            q[p] = turned(u, p, f)
        if far is not None:
            k[far] = turned(u, far, f)
            v[far] = 8.0 + rng.random((G, vdim))
        self.scale = 8.0 / dim
        self.q, self.k, self.v = (LM.rounded(a).astype(np.float64) for a in (q, k, v))
        self.qn, self.kn = LM.rounded(1 + 0.1 * rng.standard_normal(H * dim)), LM.rounded(1 + 0.1 * rng.standard_normal(G * dim))
        at = np.arange(n)
        self.qq = OL.rotate_pairs(OL.rms_norm(self.q.reshape(n, -1), self.qn, self.eps).reshape(n, H, dim), at, f)
        self.kk = OL.rotate_pairs(OL.rms_norm(self.k.reshape(n, -1), self.kn, self.eps).reshape(n, G, dim), at, f)

    def want(self, lo, hi, window=..., keep=None, f32=1, q16=False):
        """Outputs of positions lo .. hi - 1; in bf16 the keys are taken as a cache holds them (and the queries as a buffer does)."""
        kk, qq = (self.kk, self.qq) if f32 else (LM.rounded(self.kk).astype(np.float64), LM.rounded(self.qq).astype(np.float64) if q16 else self.qq)
        w, kp = self.window if window is ... else window, self.keep if keep is None else keep
        o = [OL.window_attention(qq[lo:hi, h], kk[:hi, h // (self.H // self.G)], self.v[:hi, h // (self.H // self.G)], self.scale, lo, w, kp) for h in range(self.H)]
        return np.concatenate(o, 1)

    def caches(self, dev, cap, filled, f32, noise):
        """Rows [0, filled) as stored, everything after them noise that must not be read."""
        dp, vp = up(self.dim, 8), up(self.vdim, 8)
        ck, cv = np.full((self.G, cap, dp), noise, np.float32), np.full((self.G, cap, vp), noise, np.float32)
        ck[..., self.dim:] = 0; cv[..., self.vdim:] = 0
        ck[:, :filled, :self.dim] = self.kk[:filled].transpose(1, 0, 2); cv[:, :filled, :self.vdim] = self.v[:filled].transpose(1, 0, 2)
        return dev.act(ck, f32), dev.act(cv, f32)


def edges(window, keep, p):
    """Places just inside and just outside every border of what position p sees, tile borders included."""
    c = {0, p, p - 1, 63, 64, keep - 1, keep}
    if window is not None:
        c |= {p - window + 1, p - window, p - window - 1}
    return sorted(j for j in c if 0 <= j <= p)


WINDOWS = [(None, 0), (1, 0), (7, 3), (64, 0), (40, 70), (130, 5)]


@pytest.mark.parametrize("H,G,dim,vdim,rot", ATT)
@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("before,rows", [(0, 2), (0, 70), (61, 9), (127, 66), (300, 3), (215, 130)])
def test_rotary_store_and_window_attention_rows(runtime, dev, H, G, dim, vdim, rot, f32, before, rows):
    rng = np.random.default_rng(H * 1000 + dim + before)
    n, cap = before + rows, before + rows + 3
    sz, tol, ld, ldo, dp, vp = 4 if f32 else 2, 4e-5 if f32 else 1.2e-2, up((H + G) * dim + G * vdim, 64), up(H * vdim, 64), up(dim, 8), up(vdim, 8)
    for window, keep in WINDOWS:
        for far in edges(window, keep, n - 1):
            c = AttentionCase(rng, H, G, dim, vdim, rot, n, [n - 1], far, window, keep)
            raw = np.concatenate([c.q[before:].reshape(rows, -1), c.k[before:].reshape(rows, -1), c.v[before:].reshape(rows, -1)], 1)
            ck, cv = c.caches(dev, cap, before, f32, 3.0)
            q, out, tab = dev.new(rows * H * dp * sz), dev.new(rows * ldo * sz), dev.put(rotation_table(c.rot, cap)) if rot else 0
            runtime.state_set(0, before)
            ha, da = H | G << 16, dim | vdim << 16
            runtime.launch(N.Task.make(N.TASK_ROTARY_STORE_ROWS, 0, {0: dev.act(raw, f32, ld), 1: dev.put(LM.bits(c.qn)), 2: dev.put(LM.bits(c.kn)), 3: q, 4: ck, 5: cv, 6: tab},
                                       [ha, da, cap, rows, ld, rot, f32], [c.eps]))
            runtime.launch(N.Task.make(N.TASK_WINDOW_ATTENTION_ROWS, 0, {0: q, 1: ck, 2: cv, 3: out}, [ha, da, cap, rows, f32, window or 0, keep], [c.scale]))
            assert runtime.state_get()[2] == 0
            kc = dev.get(ck, (G, cap, dp), f32)
            close(kc[:, before:n, :dim], c.kk[before:].transpose(1, 0, 2), 3e-6 if f32 else 5e-3, "stored keys")
            assert (kc[:, n:, :dim] == 3.0).all()
            want, got = c.want(before, n, f32=f32, q16=True), dev.get(out, (rows, ldo), f32)[:, :H * vdim]
            close(got, want, tol, f"window {window} keep {keep} far {far}")
            close(got[-1], want[-1], tol, f"last position, window {window} keep {keep} far {far}")
            # the cases tell a window or a kept prefix that is one off
            seen = window is None or n - 1 - far < window or far < keep
            wrong = None
            if window is not None and far in (n - 1 - window, n - window) and far >= keep:
                wrong = c.want(n - 1, n, window + (1 if not seen else -1)) if window > 1 or not seen else None
            elif window is not None and far in (keep - 1, keep) and n - 1 - far >= window:
                wrong = c.want(n - 1, n, keep=keep + (1 if not seen else -1))
            if wrong is not None:
                assert np.abs(wrong[0] - want[-1]).max() > 0.2 * np.abs(want[-1]).max(), (window, keep, far)


@pytest.mark.parametrize("H,G,dim,vdim,rot", ATT)
@pytest.mark.parametrize("f32", [0, 1])
def test_window_attention_decode(runtime, dev, H, G, dim, vdim, rot, f32):
    rng = np.random.default_rng(H + dim)
    dp, vp, tiles, sz = up(dim, 8), up(vdim, 8), -(-(H // G) // 8), 4 if f32 else 2
    for window, keep in WINDOWS:
        for pos, splits in ((0, 1), (5, 3), (64, 1), (137, 3), (400, 7)):
            for far in edges(window, keep, pos):
                cap = pos + 5
                c = AttentionCase(rng, H, G, dim, vdim, rot, pos + 1, [pos], far, window, keep)
                ck, cv = c.caches(dev, cap, pos, f32, 3.0)
                raw = np.concatenate([c.q[-1].reshape(-1), c.k[-1].reshape(-1), c.v[-1].reshape(-1)]).astype(np.float32)
                out, part, cnt = dev.new(H * vdim * 4), dev.new(G * tiles * splits * 8 * (vp + 2) * 4), dev.new(G * tiles * 4)
                t = N.Task.make(N.TASK_WINDOW_ATTENTION_DECODE, 0,
                                {0: dev.put(raw), 1: dev.put(LM.bits(c.qn)), 2: dev.put(LM.bits(c.kn)), 3: ck, 4: cv, 5: out, 6: part, 7: cnt, 8: dev.put(rotation_table(c.rot, cap)) if rot else 0},
                                [H | G << 16, dim | vdim << 16, cap, f32, splits, window or 0, keep, rot], [c.scale, c.eps])
                runtime.state_set(0, pos)
                want = c.want(pos, pos + 1, f32=f32)[0]
                for _ in range(2):                       # the split counters are left as they were found
                    runtime.launch(t)
                    assert runtime.state_get()[2] == 0
                    close(runtime.download(out, (H * vdim,), np.float32), want, 4e-5 if f32 else 8e-3, f"window {window} keep {keep} pos {pos} splits {splits} far {far}")
                kc, vc = dev.get(ck, (G, cap, dp), f32), dev.get(cv, (G, cap, vp), f32)
                close(kc[:, pos, :dim], c.kk[pos], 3e-6 if f32 else 5e-3, "stored key")
                assert np.array_equal(vc[:, pos, :vdim], c.v[pos].astype(np.float32)) and (kc[:, pos + 1:, :dim] == 3.0).all()


def memory_want(q, k, v, zi, zf, bi, bf, cap, states):
    """Outputs and, for each, the magnitude that rounding errors are a fraction of: the sums of the numerator and of the divisor taken
    with absolute values (the divisor |n . q| may come close to zero and blow up the output together with its error)."""
    out, size = np.zeros(v.shape), np.zeros(v.shape)
    for h in range(q.shape[1]):
        gi, gf = OL.soft_cap(zi[:, h] + bi[h], cap), OL.log_sigmoid(OL.soft_cap(zf[:, h] + bf[h], cap))
        out[:, h], states[h] = OL.matrix_memory(q[:, h], k[:, h], v[:, h], gi, gf, states[h])
        n, A, B, m = np.zeros(q.shape[2]), np.zeros((q.shape[2], v.shape[2])), np.zeros(q.shape[2]), 0.0
        for t in range(len(q)):
            new = max(gf[t] + m, gi[t])
            keep, add, m = np.exp(gf[t] + m - new), np.exp(gi[t] - new), new
            n, A, B = keep * n + add * k[t, h], keep * A + add * np.outer(abs(k[t, h]), abs(v[t, h])), keep * B + add * abs(k[t, h])
            size[t, h] = (A.T @ abs(q[t, h]) + abs(out[t, h]) * (B @ abs(q[t, h]))) / (max(abs(n @ q[t, h]), np.exp(-m)) + 1e-6)
    return out, size


REC = [(1, 8, 8), (3, 16, 24), (2, 40, 72), (2, 64, 64), (4, 128, 128), (1, 200, 136), (2, 256, 64), (1, 264, 16), (3, 10, 14), (1, 5, 130)]


@pytest.mark.parametrize("heads,dim,vdim", REC)
@pytest.mark.parametrize("form", ["decay", "memory"])
@pytest.mark.parametrize("dtype", ["rows32", "rows16", "decode"])
def test_recurrence(runtime, dev, heads, dim, vdim, form, dtype):
    """Portions of unequal sizes, the state carried between them: single positions, chunks of 64, borders of chunks inside and between
    portions, portions long enough to be worked on in several runs side by side.  What the state holds before position 0 is not read."""
    rng = np.random.default_rng(heads * 100 + dim)
    f32 = int(dtype != "rows16")
    portions = {"rows32": [2, 63, 66, 100], "rows16": [2, 15, 16, 64, 63, 1, 65, 700, 130, 17, 1300], "decode": [1] * 90}[dtype]
    T = sum(portions)
    q, k, v = (LM.rounded(rng.standard_normal((T, heads, n)) * s) for n, s in ((dim, 1.0), (dim, dim ** -0.5), (vdim, 1.0)))
    mem = form == "memory"
    zi, zf = (rng.standard_normal((T, heads)).astype(np.float32) * s for s in (3.0, 2.0))
    zi[T // 2] = 9.0; zi[T // 2 + 1:] -= 6.0             # a large gate in the middle: the running maximum keeps falling behind it
    bi, bf, cap, qs = LM.rounded(rng.standard_normal(heads)), LM.rounded(5 + rng.standard_normal(heads)), 7.0, 0.7
    decay = np.array([0.999, 0.9, 0.5, 0.0][:heads])
    rec = LM.MM(heads, dim, vdim, cap) if mem else LM.L(heads, dim, vdim, tuple(decay))
    if mem:
        states = [(np.zeros((dim, vdim)), np.zeros(dim), 0.0) for _ in range(heads)]
        want, size = memory_want(q * float(qs), k.astype(np.float64), v.astype(np.float64), zi.astype(np.float64), zf.astype(np.float64), bi, bf, cap, states)
    else:
        states, want, size = np.zeros((heads, dim, vdim)), np.zeros((T, heads, vdim)), np.zeros((T, heads, vdim))
        for h in range(heads):
            size[:, h] = OL.decay_recurrence(abs(q[:, h]) * float(qs), abs(k[:, h]).astype(np.float64), abs(v[:, h]).astype(np.float64), decay[h], states[h])[0]
            want[:, h], states[h] = OL.decay_recurrence(q[:, h] * float(qs), k[:, h].astype(np.float64), v[:, h].astype(np.float64), decay[h], states[h])
    slices, cell = -(-vdim // 64), TG.recurrence_cell(rec)
    state = dev.put(np.full(TG.recurrence_state(rec), np.nan, np.float32))
    ld, ldo, sz = up(heads * (2 * dim + vdim), 64), up(heads * vdim, 8), 4 if f32 else 2
    at, got = 0, []
    bias, dec = dev.put(LM.bits(np.concatenate([bi, bf]))), dev.put(np.concatenate([np.maximum(np.log(np.maximum(decay, 1e-300)), -1e4), decay]).astype(np.float32))
    need = max(TG.recurrence_scratch(rec, n) for n in portions)
    scratch = dev.new(max(need, 1) * 4)
    for n in portions:
        x = np.concatenate([a[at:at + n].reshape(n, -1) for a in (q, k, v)], 1)
        xd, out = dev.act(x, f32, ld), dev.new(n * ldo * sz)
        bufs = {0: xd, 1: xd + heads * dim * sz, 2: xd + 2 * heads * dim * sz, 6: state, 7: out}
        bufs.update({3: dev.put(np.concatenate([zi[at:at + n], zf[at:at + n]], 1)), 4: bias} if mem else {5: dec})
        runtime.state_set(0, at)
        if dtype == "decode":
            runtime.launch(N.Task.make(N.TASK_RECURRENCE_DECODE, 0, bufs, [heads, dim, vdim], [qs, cap]))
        else:
            runtime.launch(N.Task.make(N.TASK_RECURRENCE_ROWS, 0, {**bufs, 8: scratch}, [heads | f32 << 16, dim, vdim, n, ld, 2 * heads, ldo, TG.recurrence_scratch(rec, n)], [qs, cap]))
        assert runtime.state_get()[2] == 0
        got.append(dev.get(out, (n, ldo), f32)[:, :heads * vdim].reshape(n, heads, vdim)); at += n
    got = np.concatenate(got)
    err = np.abs(got - want) / ((3e-6 if f32 else 2e-5) * size + (0.0 if f32 else 2.0 ** -8) * np.abs(want) + 1e-9)
    assert err.max() <= 1.0, (np.unravel_index(err.argmax(), err.shape), err.max())
    st = runtime.download(state, (heads, slices, cell), np.float32)
    for h in range(heads):
        S = np.concatenate(list(st[h, :, :dim * 64].reshape(slices, dim, 64)), 1)[:, :vdim]
        ref = states[h][0] if mem else states[h]
        close(S, ref, 3e-5 if f32 else 1e-4, f"state {h}")
        if mem:
            close(st[h, :, dim * 64:dim * 64 + dim], np.tile(states[h][1], (slices, 1)), 3e-5 if f32 else 1e-4, "normaliser")
            assert np.abs(st[h, :, dim * 64 + dim] - states[h][2]).max() < 1e-4


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("n,group", [(64, 64), (136, 8), (130, 13), (1200, 300), (2048, 2048)])
def test_norm_gate_rows(runtime, dev, n, group, f32):
    rng = np.random.default_rng(n)
    M, eps = 3, 1e-3
    o, g, w = LM.rounded(rng.standard_normal((M, n)) * 4), LM.rounded(rng.standard_normal((M, n))), LM.rounded(1 + 0.2 * rng.standard_normal(n))
    out = dev.new(M * up(n, 64) * 4)
    runtime.launch(N.Task.make(N.TASK_NORM_GATE_ROWS, 0, {0: dev.act(o, f32, n + 6), 1: dev.put(LM.bits(w)), 2: dev.act(g, f32, n + 2), 3: out}, [n, group, M, n + 6, n + 2, up(n, 64), f32], [eps]))
    want = OL.rms(o.astype(np.float64).reshape(M, -1, group), eps).reshape(M, n) * w * OL.sigmoid(g.astype(np.float64))
    close(dev.get(out, (M, up(n, 64)), f32)[:, :n], want, 3e-6 if f32 else 5e-3)


@pytest.mark.parametrize("rows,ks,gseg,group", [(8, (8,), 0, 4), (75, (132, 42, 37), 1, 42), (300, (40, 1000), 0, 8), (2048, (2048, 2048, 4096), 1, 2048), (513, (3000, 64, 600), 2, 60)])
def test_segment_linear(runtime, dev, rows, ks, gseg, group):
    rng = np.random.default_rng(rows)
    eps, xs = 1e-3, [rng.standard_normal(k).astype(np.float32) for k in ks]
    W = [LM.bits(rng.standard_normal((rows, k))) for k in ks]
    w, gate = LM.rounded(1 + 0.2 * rng.standard_normal(ks[gseg])), rng.standard_normal(ks[gseg]).astype(np.float32)
    for g in (gseg, -1):
        y = dev.new(len(ks) * rows * 4)
        bufs = {6: y, 7: dev.put(LM.bits(w)), 8: dev.put(gate)}
        for s, (x, m) in enumerate(zip(xs, W)):
            bufs.update({2 * s: dev.put(x), 2 * s + 1: rows_weight(runtime, m)})
        runtime.launch(N.Task.make(N.TASK_SEGMENT_LINEAR, 0, bufs, [rows, len(ks), *ks, *[0] * (3 - len(ks)), g, group], [eps]))
        got = runtime.download(y, (len(ks), rows), np.float32)
        for s, (x, m) in enumerate(zip(xs, W)):
            x = x.astype(np.float64)
            if s == g:
                x = OL.rms(x.reshape(-1, group), eps).reshape(-1) * w * OL.sigmoid(gate.astype(np.float64))
            close(got[s], LM.values(m).astype(np.float64) @ x, 4e-6, f"product {s}")


@pytest.mark.parametrize("k,silu,plain,pairs", [(8, 0, 4, 3), (75, 20, 32, 37), (1000, 64, 96, 200), (2048, 1000, 1024, 900), (4500, 10, 32, 8)])
@pytest.mark.parametrize("np_,nn", [(0, 0), (1, 0), (2, 0), (3, 2), (3, 3)])
def test_norm_linear_of_a_block(runtime, dev, k, silu, plain, pairs, np_, nn):
    """The prologue (several pending outputs, layer norm) and the end (silu range, gate/up pairs, a factor) of the joint projection."""
    rng = np.random.default_rng(k + np_)
    eps, n, limit = 1e-3, plain + 2 * pairs, 0.9
    x, y = (rng.standard_normal(k) + 9).astype(np.float32), rng.standard_normal((3, k)).astype(np.float32)
    post, w, b = (LM.rounded(1 + 0.2 * rng.standard_normal(s)) for s in ((3, k), k, k))
    W = LM.bits(rng.standard_normal((n, k)) * k ** -0.5)
    out, xo, ho, wid = dev.new(n * 4), dev.new(k * 4), dev.new(k * 4), rows_weight(runtime, W)
    bufs = {0: dev.put(x), 4: xo, 5: dev.put(LM.bits(w)), 6: wid, 7: out, 8: ho, 11: dev.put(LM.bits(b))}
    if np_:
        bufs.update({1: dev.put(y), 2: dev.put(LM.bits(post))})
    runtime.launch(N.Task.make(N.TASK_NORM_LINEAR, 0, bufs, [k, n, N.ACT_SILU if silu else 0, 0, np_, nn, plain, silu], [eps, 0.5, limit]))
    xn = x.astype(np.float64)
    for j in range(np_):
        xn = xn + (0.5 * OL.rms_norm(y[j].astype(np.float64), post[j], eps) if j < nn else y[j])
    h = OL.layer_norm(xn, w, b, eps)
    z = LM.values(W).astype(np.float64) @ h
    got = runtime.download(out, (n,), np.float32)
    close(runtime.download(xo, (k,), np.float32), xn, 1e-6, "x")
    close(runtime.download(ho, (k,), np.float32), h, 1e-5, "h")
    if silu:
        close(got[:silu], OL.silu(z[:silu]), 2e-5, "silu")
    close(got[silu:plain], z[silu:plain], 2e-5, "plain")
    close(got[plain:plain + pairs], OL.clamped_glu(z[plain::2], z[plain + 1::2], limit), 2e-5, "pairs")
    runtime.launch(N.Task.make(N.TASK_NORM_LINEAR, 0, bufs, [k, n, 0, 0, np_, nn, 0, 0], [eps, 0.5, 0.0, 2.5]))
    close(runtime.download(out, (n,), np.float32), 2.5 * z, 2e-5, "factor")


def test_bad_block_arguments_are_refused(runtime, dev):
    b = dev.new(1 << 14)
    for t in (N.Task.make(N.TASK_RECURRENCE_DECODE, 0, {i: b for i in (0, 1, 2, 5, 6, 7)}, [1, 513, 8], [1.0, 0.0]),
              N.Task.make(N.TASK_WINDOW_ATTENTION_ROWS, 0, {i: b for i in range(4)}, [1 | 1 << 16, 8 | 8 << 16, 16, 2, 1, -1, 0], [1.0]),
              N.Task.make(N.TASK_ROTARY_STORE_ROWS, 0, {i: b for i in range(6)}, [1 | 1 << 16, 8 | 8 << 16, 16, 2, 64, 4, 1], [1e-6]),       # rotation without a table
              N.Task.make(N.TASK_BLOCK_NORM_ROWS, 0, {0: b, 5: b, 6: b}, [64, 2, 1, 64, 64, 1, 0], [1e-6]),
              N.Task.make(N.TASK_NORM_GATE_ROWS, 0, {i: b for i in range(4)}, [64, 7, 2, 64, 64, 64, 1], [1e-6])):
        with pytest.raises(N.FusekitError):
            runtime.launch(t)


# ------------------------------------------------------------------ whole models
PORTIONS = {"whole": None, "twos": [2], "mixed": [7, 2, 33, 1, 64, 3], "single": [1]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(LM.PARALLEL_SPECS))
def test_portions_of_a_prompt_match_the_oracle(runtime, name, dtype):
    s = LM.PARALLEL_SPECS[name]
    t = LM.random_tensors(s, 5)
    toks = np.random.default_rng(2).integers(0, s.vocab, 170)
    want = LM.oracle(s, t).forward(toks)
    e = LM.engine(s, t, 190, dtype, runtime=runtime, max_rows=120)
    other, slots = e.open_sequence(), set()
    other.append(toks[::-1][:20])
    for how, sizes in PORTIONS.items():
        seq, got, p, j = e.open_sequence(), [], 0, 0
        slots.add(seq.slot)
        while p < len(toks):
            n = len(toks) if sizes is None else min(sizes[j % len(sizes)], len(toks) - p)
            got.append(seq.append(toks[p:p + n], list(range(n)))); p += n; j += 1
        seq.close()
        check_logits(np.concatenate(got), want, dtype, f"{name} {how}")
    assert len(slots) == 1 and other.slot not in slots
    w2 = LM.oracle(s, t).forward(toks[::-1][:25])
    check_logits(other.append(toks[::-1][20:25], [0, 1, 2, 3, 4]), w2[20:], dtype, "kept sequence")
    other.close()


def test_interleaved_sequences_do_not_touch_each_other(runtime):
    """Unequal sequences in turns, some ending and their slots used again, each against itself alone."""
    s = LM.PARALLEL_SPECS["mixed"]
    t = LM.random_tensors(s, 11)
    e = LM.engine(s, t, 120, "float32", runtime=runtime)
    rng = np.random.default_rng(4)
    texts = [rng.integers(0, s.vocab, n) for n in (100, 7, 55, 1, 30, 90)]
    want = [LM.oracle(s, t).forward(x) for x in texts]
    live, waiting, done = {}, list(range(len(texts))), 0
    while done < len(texts):
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = [e.open_sequence(), 0]
        for i in list(live):
            seq, p = live[i]
            n = min(int(rng.integers(1, 30)), len(texts[i]) - p)
            check_logits(seq.append(texts[i][p:p + n], list(range(n))), want[i][p:p + n], "float32", f"sequence {i} at {p}")
            live[i][1] += n
            if p + n == len(texts[i]):
                seq.close(); del live[i]; done += 1
    assert len(e.caches) == 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_and_long_decoding(runtime, dtype):
    """A prompt long enough that the recurrences work on several runs of chunks, then hundreds of decoded positions: a window passes
    over them and a slow state keeps the beginning."""
    s = LM.parallel_spec([LM.LayerSpec(LM.P(LM.windowed(2, 1, 16, 16, 0.4, 90, 4, 16), LM.L(2, 16, 32, (0.9, 0.998))), LM.G(32, 1.0)), LM.LayerSpec(LM.MM(2, 16, 32, 9.0), LM.G(16, 2.0))],
                         hidden=64, vocab=120)
    t = LM.random_tensors(s, 4)
    toks = np.random.default_rng(3).integers(0, s.vocab, 1500)
    want = LM.oracle(s, t).forward(toks)
    e = LM.engine(s, t, 1500, dtype, runtime=runtime)
    seq = e.open_sequence()
    check_logits(seq.append(toks[:1100], list(range(1100))), want[:1100], dtype, "prompt")
    got = np.concatenate([seq.append(toks[i:i + 1], [0]) for i in range(1100, 1500)])
    check_logits(got, want[1100:], dtype, "decoded")
    seq.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_at_the_edge_of_what_is_seen_decides_the_output(runtime, dtype):
    """Marker and asking token of one attention layer whose linear attention is silenced by a small norm weight: logits must change with the
    marker exactly where it is seen -- through prompts, portions and decoding."""
    W, K = 37, 5
    s = LM.parallel_spec([LM.LayerSpec(LM.P(LM.windowed(2, 1, 16, 24, 1.2, W, K, None), LM.L(1, 8, 8, (0.01,))), None)], hidden=64, vocab=50)
    t = LM.random_tensors(s, 9)
    emb = LM.values(t["embed"]).copy()
    emb[:, :2] = 0.0
    emb[7, 0] = 12.0; emb[8, 1] = 12.0                   # 7: marker (keys), 8: asks for it (queries)
    t["embed"] = LM.bits(emb)
    q, k = LM.values(t["l0.mix.left.q"]).copy(), LM.values(t["l0.mix.left.k"]).copy()
    u = np.random.default_rng(0).standard_normal(16)
    q[:, 1] = np.tile(u, 2) * 3; k[:, 0] = u * 3
    t["l0.mix.left.q"], t["l0.mix.left.k"] = LM.bits(q), LM.bits(k)
    t["l0.mix.right.out"], t["l0.mix.left.out"] = LM.bits(np.full(64, 0.01)), LM.bits(3 * LM.values(t["l0.mix.left.out"]))
    n = 150
    e = LM.engine(s, t, n + 4, dtype, runtime=runtime)
    for far, seen in ((0, 1), (K - 1, 1), (K, 0), (n - 1 - W, 0), (n - W, 1), (n - 2, 1), (64, 0)):
        toks = np.random.default_rng(far).integers(10, s.vocab, n); toks[far] = 7; toks[-1] = 8
        without = toks.copy(); without[far] = 11
        want, blind = (LM.oracle(s, t).forward(x)[-1:] for x in (toks, without))
        change = LM.logit_error(blind, want)[0]
        assert change > 0.3 if seen else change < 0.01, far
        for cut in (0, n - 1, n - 2, 64):
            seq = e.open_sequence()
            if cut:
                seq.append(toks[:cut])
            got = seq.append(toks[cut:], [n - cut - 1])
            seq.close()
            assert LM.logit_error(got, want)[0] < (F32_TOL if dtype == "float32" else BF16_TOL), (far, cut)


@pytest.mark.parametrize("name", ["mixed", "odd-sizes"])
def test_greedy_and_sampled_generation(runtime, tmp_path, name):
    s = LM.PARALLEL_SPECS[name]
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


def test_command_line(tmp_path, capsys):
    from fusekit_b200.generate import main
    s = LM.PARALLEL_SPECS["memory-first"]
    t = LM.random_tensors(s, 8)
    LM.write_model(tmp_path / "m", s, t)
    o, want, toks = LM.oracle(s, t), [], [3, 1, 4]
    for _ in range(6):
        toks = [int(np.argmax(o.forward(toks)[-1]))]; want += toks
    assert main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--prompt", "3,1,4", "--max-tokens", "6"]) == 0
    assert [int(v) for v in capsys.readouterr().out.split(",")] == want
    args = ["--config", "tiny-kakunex", "--prompt", "3,1,4", "--max-tokens", "6"]
    assert main(args) == 0 and main(args + ["--temperature", "0.8", "--top-k", "1"]) == 0
    a, b = capsys.readouterr().out.split()
    assert a == b and len(a.split(",")) == 6


def test_registered_shape_through_attach(runtime):
    import json
    e = attach(LAYERED_CONFIGS["tiny-kakunex"], 64, runtime=runtime)
    e.load_synthetic()
    first = e.prefill([5, 9, 2, 44])
    a, _ = e.generate(first, 4, 20)
    e.prefill([5, 9, 2, 44])
    e.capture_json(json.dumps(e.task_graph()))
    b, _ = e.generate(first, 4, 20)
    assert a.tolist() == b.tolist() and len(set(a.tolist())) > 1
    assert TG.K_RECDEC in [t.kind for t in e.replay]


def test_a_state_is_continued_where_it_stands(runtime):
    s = LM.PARALLEL_SPECS["one-layer"]
    t = LM.random_tensors(s)
    e = LM.engine(s, t, 16, runtime=runtime)
    want = LM.oracle(s, t).forward([1, 2, 3, 4, 5])
    e.step([1, 2, 3], 0)
    for call in (lambda: e.step([4], 2), lambda: e.step([4, 5], 4), lambda: e.decode_chunk(1, 4, 2), lambda: e.step([1] * 14, 3), lambda: e.step([s.vocab], 3)):
        with pytest.raises(ValueError):
            call()
    check_logits(e.step([4, 5], 3, [0, 1]), want[3:], "float32")
    check_logits(e.step([1, 2], 0, [0, 1]), want[:2], "float32", "started again")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_stream_after_every_layer(runtime, dtype):
    s = LM.PARALLEL_SPECS["mixed"]
    t = LM.random_tensors(s, 2)
    toks = np.random.default_rng(0).integers(0, s.vocab, 30)
    o = LM.oracle(s, t)
    o.forward(toks)
    e = LM.engine(s, t, 40, dtype, runtime=runtime)
    e.step(toks[:-1], 0)
    e.step(toks[-1:], 29)
    for i, (a, b) in enumerate(zip(e.residual_stream()[1:], o.residuals)):
        close(a, b[-1], 2e-5 if dtype == "float32" else 3e-2, f"after layer {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_writes_the_asked_logits(runtime, tmp_path, dtype):
    from fusekit_b200.trace import TraceRunner
    s = LM.PARALLEL_SPECS["mixed"]
    t = LM.random_tensors(s, 6)
    LM.write_model(tmp_path / "m", s, t)
    e, ck = CK.load_engine(str(tmp_path / "m"), 64, dtype=dtype, runtime=runtime)
    toks = np.random.default_rng(1).integers(0, s.vocab, 30).tolist()
    want = LM.oracle(s, t).forward(toks)
    r = TraceRunner(e, str(tmp_path))
    r.step({"step": 0, "entries": [{"id": "a", "tokens": toks[:20], "want": [3, 19]}], "end": []})
    r.step({"step": 1, "entries": [{"id": "a", "tokens": toks[20:28], "want": []}], "end": []})
    r.step({"step": 2, "entries": [{"id": "a", "tokens": toks[28:], "want": [1]}], "end": ["a"]})
    r.step({"step": 3, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}], "end": ["b"]})
    assert not (tmp_path / "1.f32").exists() and not r.live and len(e.caches) == 1
    for step, rows in ((0, [3, 19]), (2, [29]), (3, [0])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), s.vocab)
        assert LM.logit_error(got, want[rows]).max() < (F32_TOL if dtype == "float32" else 4 * BF16_TOL)
    ck.close()
