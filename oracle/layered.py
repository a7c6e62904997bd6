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
