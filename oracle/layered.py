"""Plain NumPy restatement of the layered decoders (``model_spec.LayeredSpec``): one slow function per mechanism, written
from the equations and sharing no code with the product path.  Test infrastructure, like the rest of this folder.

Notation: x is the residual stream [T, D]; a layer adds norm(mixer(norm(x))) and then norm(ff(norm(x))).  Everything is
computed in one floating type (float64 by default), so results differ from a correct device run by rounding only.
"""
from __future__ import annotations

import numpy as np


def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def softmax_attention(q, k, v, scale, pos0):
    """One head: q [Tq, d] at positions pos0 .., keys k [Tk, d] and values v [Tk, dv] at positions 0 ..; causal."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for i in range(q.shape[0]):
        n = pos0 + i + 1
        s = (k[:n] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[:n]
    return out


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def differential_combine(a1, a2, lam, diff, eps):
    """a1 - lambda a2, unit root mean square over the head's values, times (1 - diff)."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def route(logits, top):
    """Indices of the `top` largest logits (lowest index first among equals) and the softmax over just those."""
    idx = np.argsort(-logits, axis=-1, kind="stable")[..., :top]
    z = np.take_along_axis(logits, idx, -1)
    p = np.exp(z - z.max(-1, keepdims=True))
    return idx, p / p.sum(-1, keepdims=True)


def expert(w_up, w_down, h):
    return relu_squared(h @ w_up.T) @ w_down.T


class LayeredOracle:
    """``spec``: a LayeredSpec (only its numbers are read); ``tensors``: name -> array.  Sequences carry their own keys and
    values per layer run, so a prompt may arrive in any portions."""

    def __init__(self, spec, tensors, dtype=np.float64):
        self.spec, self.dt = spec, dtype
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.pos, self.kv = 0, {}

    def attention(self, i, run, h):
        m, t, eps = self.spec.layers[i].mixer, self.t, self.spec.eps
        p = f"l{i}.mix."
        T, H, G, d, dv = h.shape[0], m.heads, m.kv_heads, m.dim, m.vdim
        maps = 2 if m.diff is not None else 1
        q = (h @ t[p + "q"].T).reshape(T, H, maps, d)
        k = (h @ t[p + "k"].T).reshape(T, G, maps, d)
        v = (h @ t[p + "v"].T).reshape(T, G, dv)
        q, k = rms_norm(q, t[p + "q.norm"], eps), rms_norm(k, t[p + "k.norm"], eps)
        if run in self.kv:
            k, v = np.concatenate([self.kv[run][0], k]), np.concatenate([self.kv[run][1], v])
        self.kv[run] = (k, v)
        gate = sigmoid(h @ t[p + "g"].T)
        o = np.zeros((T, H, dv), self.dt)
        for hh in range(H):
            g = hh // (H // G)
            a = [softmax_attention(q[:, hh, j], k[:, g, j], v[:, g], m.scale, self.pos) for j in range(maps)]
            if maps == 2:
                lam = differential_lambda(*(t[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m.diff)
                a = [differential_combine(a[0], a[1], lam, m.diff, eps)]
            o[:, hh] = a[0] * gate[:, hh:hh + 1]
        return o.reshape(T, H * dv) @ t[p + "o"].T

    def feed_forward(self, i, h):
        f, t = self.spec.layers[i].mlp, self.t
        p = f"l{i}.mlp."
        idx, w = route(h @ t[p + "router"].T, f.top)
        y = np.zeros_like(h)
        for r in range(h.shape[0]):
            for j in range(f.top):
                e = f"{p}e{idx[r, j]}."
                y[r] += w[r, j] * expert(t[e + "up"], t[e + "down"], h[r:r + 1])[0]
        if f.shared_ff:
            y = y + expert(t[p + "shared.up"], t[p + "shared.down"], h)
        return y

    def runs(self):
        """(layer, pass is a repetition and this is its first layer) in execution order."""
        lp, n = self.spec.loop, len(self.spec.layers)
        if lp is None:
            return [(i, False) for i in range(n)]
        out = [(i, False) for i in range(lp.start)]
        for k in range(lp.times):
            out += [(i, k > 0 and i == lp.start) for i in range(lp.start, lp.stop)]
        return out + [(i, False) for i in range(lp.stop, n)]

    def forward(self, tokens):
        """Logits [T, V] of the next portion of the sequence; ``self.residuals`` keeps x after every layer run."""
        t, eps = self.t, self.spec.eps
        emb = t["embed"][np.asarray(tokens, np.int64)]
        x, self.residuals = emb.copy(), []
        for run, (i, again) in enumerate(self.runs()):
            if again:
                x = x + emb
            n = f"l{i}."
            x = x + rms_norm(self.attention(i, run, rms_norm(x, t[n + "norm1"], eps)), t[n + "norm1b"], eps)
            if self.spec.layers[i].mlp is not None:
                x = x + rms_norm(self.feed_forward(i, rms_norm(x, t[n + "norm2"], eps)), t[n + "norm2b"], eps)
            self.residuals.append(x)
        self.pos += len(tokens)
        return rms_norm(x, t["final.norm"], eps) @ t["head"].T


# ---------------------------------------------------------------- parallel blocks: layer norm, rotation, windows, recurrences
def layer_norm(x, w, b, eps):
    """Mean and variance along the last axis; eps inside the root."""
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def silu(z):
    return z * sigmoid(z)


def clamped_glu(gate, up, limit):
    """s(g) (u + 1) with s(g) = g sigmoid(1.702 g), the gate bounded from above and the up value on both sides."""
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def rotation_frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair; ``scaling`` = (factor, low, high, original) stretches the long wavelengths."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high, original = scaling
            wave = 2.0 * np.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out)


def rotate_pairs(x, positions, freqs):
    """x [T, heads, d]: neighbours (2i, 2i + 1) turned by position * freqs[i]; dimensions past the last pair are kept."""
    out = x.copy()
    for i, f in enumerate(freqs):
        a = np.asarray(positions, np.float64) * f
        c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_attention(q, k, v, scale, pos0, window=None, keep_first=0):
    """One head, as softmax_attention over the newest ``window`` positions up to the query and the first ``keep_first`` of all."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for i in range(q.shape[0]):
        p = pos0 + i
        j = np.arange(p + 1)
        see = j[(p - j < window) | (j < keep_first)] if window is not None else j
        s = (k[see] @ q[i]) * scale
        e = np.exp(s - s.max())
        out[i] = (e / e.sum()) @ v[see]
    return out


def decay_recurrence(q, k, v, decay, state):
    """One head: S <- decay S + k v^T, o = S^T q.  ``state``: S [dim, vdim].  Returns (o, S)."""
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        state = decay * state + np.outer(k[t], v[t])
        out[t] = state.T @ q[t]
    return out, state


def matrix_memory(q, k, v, log_i, log_f, state):
    """One head of a matrix memory with exponential gates kept in range by a running maximum.  ``state``: (S, n, m)."""
    S, n, m = state
    out = np.zeros((q.shape[0], v.shape[1]), q.dtype)
    for t in range(q.shape[0]):
        new = max(log_f[t] + m, log_i[t])
        keep, add = np.exp(log_f[t] + m - new), np.exp(log_i[t] - new)
        S, n, m = keep * S + add * np.outer(k[t], v[t]), keep * n + add * k[t], new
        out[t] = (S.T @ q[t]) / (max(abs(n @ q[t]), np.exp(-m)) + 1e-6)
    return out, (S, n, m)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


class ParallelBlockOracle:
    """Layers in which the mixer and the feed-forward read one layer norm and are added together.  Same interface as
    LayeredOracle; only the numbers of ``spec`` are read, and a mixer is told by the fields it has."""

    def __init__(self, spec, tensors, dtype=np.float64):
        self.spec, self.dt = spec, dtype
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.pos, self.mem = 0, {}

    def attention(self, key, p, m, h):
        t, eps, T = self.t, self.spec.eps, h.shape[0]
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        q = rms_norm(h @ t[p + "q"].T, t[p + "q.norm"], eps).reshape(T, H, d)
        k = rms_norm(h @ t[p + "k"].T, t[p + "k.norm"], eps).reshape(T, G, d)
        v = (h @ t[p + "v"].T).reshape(T, G, dv)
        if m.rotary is not None:
            r = m.rotary
            s = None if r.scaling is None else (r.scaling.factor, r.scaling.low, r.scaling.high, r.scaling.original)
            f = rotation_frequencies(r.dims, r.base, s)
            at = self.pos + np.arange(T)
            q, k = rotate_pairs(q, at, f), rotate_pairs(k, at, f)
        if key in self.mem:
            k, v = np.concatenate([self.mem[key][0], k]), np.concatenate([self.mem[key][1], v])
        self.mem[key] = (k, v)
        o = [window_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m.scale, self.pos, m.window, m.keep_first) for i in range(H)]
        return np.concatenate(o, 1) @ t[p + "o"].T

    def lightning(self, key, p, m, h):
        t, T = self.t, h.shape[0]
        q, k, v = (silu(h @ t[p + n].T).reshape(T, m.heads, -1) for n in "qkv")
        S, o = self.mem.get(key, np.zeros((m.heads, m.dim, m.vdim), self.dt)).copy(), []
        for i in range(m.heads):
            y, S[i] = decay_recurrence(q[:, i], k[:, i], v[:, i], m.decay[i], S[i])
            o.append(y)
        self.mem[key] = S
        o = rms_norm(np.concatenate(o, 1), t[p + "norm"], self.spec.eps) * sigmoid(h @ t[p + "g"].T)
        return o @ t[p + "o"].T

    def mlstm(self, key, p, m, h):
        t, T, eps = self.t, h.shape[0], self.spec.eps
        q = (h @ t[p + "q"].T).reshape(T, m.heads, m.dim) * m.dim ** -0.5
        k, v = (h @ t[p + "k"].T).reshape(T, m.heads, m.dim), (h @ t[p + "v"].T).reshape(T, m.heads, m.vdim)
        gi = soft_cap(h @ t[p + "i"].T + t[p + "i.b"], m.gate_cap)
        gf = log_sigmoid(soft_cap(h @ t[p + "f"].T + t[p + "f.b"], m.gate_cap))
        st = self.mem.get(key) or [(np.zeros((m.dim, m.vdim), self.dt), np.zeros(m.dim, self.dt), 0.0) for _ in range(m.heads)]
        o, new = [], []
        for i in range(m.heads):
            y, s = matrix_memory(q[:, i], k[:, i], v[:, i], gi[:, i], gf[:, i], st[i])
            o.append(rms(y, eps)); new.append(s)
        self.mem[key] = new
        return (np.concatenate(o, 1) * t[p + "norm"] * sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T

    def mixer(self, i, m, h):
        p = f"l{i}.mix."
        if hasattr(m, "left"):
            a = self.attention((i, "left"), p + "left.", m.left, h)
            b = self.lightning((i, "right"), p + "right.", m.right, h)
            return 0.5 * (rms_norm(a, self.t[p + "left.out"], self.spec.eps) + rms_norm(b, self.t[p + "right.out"], self.spec.eps))
        return self.mlstm(i, p, m, h)

    def feed_forward(self, i, f, h):
        p = f"l{i}.mlp."
        return clamped_glu(h @ self.t[p + "gate"].T, h @ self.t[p + "up"].T, f.limit) @ self.t[p + "down"].T

    def forward(self, tokens):
        t, eps = self.t, self.spec.eps
        x, self.residuals = t["embed"][np.asarray(tokens, np.int64)].copy(), []
        for i, l in enumerate(self.spec.layers):
            h = layer_norm(x, t[f"l{i}.norm1"], t[f"l{i}.norm1.b"], eps)
            y = self.mixer(i, l.mixer, h)
            x = x + (y if l.mlp is None else y + self.feed_forward(i, l.mlp, h))
            self.residuals.append(x)
        self.pos += len(tokens)
        return layer_norm(x, t["final.norm"], t["final.norm.b"], eps) @ t["embed"].T * self.spec.logit_scale
