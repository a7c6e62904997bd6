"""Decoder shapes of the benchmark configs and the naming of their seeded tensors.

The reference learns these from ``config.json`` (``ModelMeta::from_config_file``,
src/fusion/ir.rs:604-749) and from the traced graph; capture needs MLX, so the five
benchmark shapes are stated here directly.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, replace

MASK64 = (1 << 64) - 1


@dataclass(frozen=True)
class ModelSpec:
    name: str
    arch: str                 # "qwen2" | "gemma3"
    n_layers: int
    hidden: int
    n_q: int
    n_kv: int
    head_dim: int
    inter: int
    vocab: int
    bits: int = 4             # 4 / 8 affine group-64, 16 = plain bf16
    eps: float = 1e-6
    theta: float = 1e6        # RoPE base of global-attention layers
    theta_local: float = 1e4  # RoPE base of sliding-window layers
    window: int = 0           # sliding window (0: every layer global)
    global_every: int = 1     # with a window: every Nth layer is global
    seed: int = 20240531

    @property
    def qkv_bias(self) -> bool:
        return self.arch == "qwen2"

    @property
    def act(self) -> int:
        return 1 if self.arch == "gemma3" else 0

    def is_sliding(self, layer: int) -> bool:
        return self.window > 0 and ((layer + 1) % self.global_every != 0)

    def layer_capacity(self, layer: int, capacity: int) -> int:
        return self.window if self.is_sliding(layer) else capacity

    def layer_theta(self, layer: int) -> float:
        return self.theta_local if self.is_sliding(layer) else self.theta

    def with_bits(self, bits: int) -> "ModelSpec":
        return replace(self, bits=bits)

    # ---- algorithmic bytes (what a decode step must read from HBM) ----
    def linear_bytes(self, k: int, n: int, residual: bool = False) -> int:
        """bytes(qmatvec K->N) = N*K*bits/8 + 2*N*(K/64)*2 + 2K + 2N (+2N with a residual)."""
        w = n * k * self.bits // 8 + (0 if self.bits == 16 else 2 * n * (k // 64) * 2)
        return w + 2 * k + 2 * n + (2 * n if residual else 0)

    def weight_bytes_per_token(self) -> int:
        h, i, qkv = self.hidden, self.inter, (self.n_q + 2 * self.n_kv) * self.head_dim
        per_layer = (self.linear_bytes(h, qkv) + self.linear_bytes(self.n_q * self.head_dim, h, True)
                     + 2 * self.linear_bytes(h, i) + self.linear_bytes(i, h, True))
        return self.n_layers * per_layer + self.linear_bytes(h, self.vocab)

    def kv_bytes_per_token(self, ctx: int) -> int:
        tot = 0
        for l in range(self.n_layers):
            n = min(ctx, self.window) if self.is_sliding(l) else ctx
            tot += 2 * self.n_kv * self.head_dim * 2 * n
        return tot

    def bytes_per_token(self, ctx: int) -> int:
        return self.weight_bytes_per_token() + self.kv_bytes_per_token(ctx)


# ---------------------------------------------------------------- decoders described layer by layer
@dataclass(frozen=True)
class FrequencyScaling:
    """Stretching of slow rotations: wavelengths above original / low turn ``factor`` times slower, those below original / high
    keep their speed, those between are blended linearly in original / wavelength."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of a head, neighbours (2i, 2i + 1) forming pairs."""
    dims: int
    base: float
    scaling: FrequencyScaling | None = None

    def frequencies(self) -> list:
        """Radians per position of every pair."""
        out, s = [], self.scaling
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if s is not None:
                wave = 2.0 * math.pi / f
                if wave > s.original / s.low:
                    f /= s.factor
                elif wave >= s.original / s.high:
                    w = (s.original / wave - s.low) / (s.high - s.low)
                    f = (1.0 - w) * f / s.factor + w * f
            out.append(f)
        return out


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention with RMS-normed queries and keys.  ``diff`` set: differential attention -- every head has two query/key
    maps over the same values, combined as a1 - lambda a2.  ``norm``: "head" (every (sub-)head by itself, one weight of size dim)
    or "projection" (all rows at once, a weight for every row).  ``gate``: a sigmoid output gate per head.  ``window`` set:
    a position sees the newest ``window`` positions up to itself and the first ``keep_first`` of the sequence."""
    heads: int
    kv_heads: int
    dim: int                  # query/key size of a map
    vdim: int
    scale: float              # score = (q . k) * scale
    diff: float | None = None
    norm: str = "head"
    gate: bool = True
    rotary: RotarySpec | None = None
    window: int | None = None
    keep_first: int = 0

    @property
    def maps(self) -> int:
        return 1 if self.diff is None else 2

    @property
    def q_rows(self) -> int:
        return self.heads * self.maps * self.dim

    @property
    def k_rows(self) -> int:
        return self.kv_heads * self.maps * self.dim

    @property
    def v_rows(self) -> int:
        return self.kv_heads * self.vdim

    @property
    def rows(self) -> int:    # q | k | v | gate, the fused projection
        return self.q_rows + self.k_rows + self.v_rows + (self.heads if self.gate else 0)

    @property
    def out_rows(self) -> int:
        return self.heads * self.vdim

    def visible(self, ctx: int) -> int:
        """Keys that a position with ``ctx`` positions up to and including itself sees."""
        return ctx if self.window is None else min(ctx, self.window + min(self.keep_first, max(ctx - self.window, 0)))

    def check(self):
        r = self.rotary
        return (min(self.heads, self.kv_heads, self.dim, self.vdim) >= 1 and self.heads % self.kv_heads == 0 and self.norm in ("head", "projection")
                and (self.window is None or self.window >= 1) and self.keep_first >= 0 and (r is None or (0 <= r.dims <= self.dim and r.dims % 2 == 0)))


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, with q, k, v behind a silu; the joined heads
    are RMS-normed together and gated."""
    heads: int
    dim: int
    vdim: int
    decay: tuple

    @property
    def qkv_rows(self) -> int:
        return self.heads * (2 * self.dim + self.vdim)

    @property
    def out_rows(self) -> int:
        return self.heads * self.vdim

    @property
    def norm_group(self) -> int:      # values that are normed together
        return self.heads * self.vdim

    def check(self):
        return min(self.heads, self.dim, self.vdim) >= 1 and len(self.decay) == self.heads and all(0.0 <= d <= 1.0 for d in self.decay)


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Matrix memory with exponential input and forget gates (mLSTM), kept in range by a running maximum of their logarithms, and
    a normaliser; every head's output is RMS-normed by itself, scaled and gated.  Gate logits are capped at +-gate_cap."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @property
    def qkv_rows(self) -> int:
        return self.heads * (2 * self.dim + self.vdim)

    @property
    def out_rows(self) -> int:
        return self.heads * self.vdim

    @property
    def norm_group(self) -> int:
        return self.vdim

    def check(self):
        return min(self.heads, self.dim, self.vdim) >= 1 and self.gate_cap > 0.0


@dataclass(frozen=True)
class ParallelMixerSpec:
    """Attention and linear attention side by side on one input: half the sum of their RMS-normed outputs."""
    left: AttentionSpec
    right: LightningSpec

    def check(self):
        return self.left.check() and self.right.check() and self.left.maps == 1 and not self.left.gate


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of ``experts`` feed-forward layers W_down relu(W_up h)^2, ``top`` per token weighted by the softmax over the
    chosen router logits, plus a shared one of size ``shared_ff`` (0: none)."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0

    def check(self):
        return 1 <= self.top <= self.experts and self.ff >= 1 and self.shared_ff >= 0


@dataclass(frozen=True)
class ClampedGluSpec:
    """Gated feed-forward: with g = min(W_gate h, limit) and u = W_up h clamped to +-limit, W_down (g sigmoid(1.702 g) (u + 1))."""
    ff: int
    limit: float

    def check(self):
        return self.ff >= 1 and self.limit > 0.0


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | ParallelMixerSpec | MatrixMemorySpec
    mlp: MoeSpec | ClampedGluSpec | None = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row; the embedding output is added to x before each repetition."""
    start: int
    stop: int
    times: int


BLOCK_COLUMNS = 32        # the joint projection of a parallel block changes its output form at multiples of this many rows


def round_up(v: int, m: int) -> int:
    return (v + m - 1) // m * m


@dataclass(frozen=True)
class BlockLayout:
    """Rows of a parallel block's joint projection, everything that reads the layer's normed input: ``parts`` (name, first row,
    rows); rows [0, silu) pass a silu, [0, plain) are the mixer's, [plain, exact) logits of recurrence gates (kept in fp32), the
    rest alternates gate and up rows of the feed-forward.  ``sources``: (tensor leaf, first row, rows)."""
    parts: dict
    sources: tuple
    silu: int
    plain: int
    exact: int
    rows: int
    out_rows: int             # with every gate / up pair folded into one value


def block_layout(layer: LayerSpec) -> BlockLayout:
    m, f, parts, src, at = layer.mixer, layer.mlp, {}, [], 0

    def put(part, *leaves):
        nonlocal at
        parts[part] = at
        for leaf, rows in leaves:
            src.append((leaf, at, rows)); at += rows

    silu = 0
    if isinstance(m, ParallelMixerSpec):
        l, r = m.left, m.right
        put("recurrence", ("mix.right.q", r.heads * r.dim), ("mix.right.k", r.heads * r.dim), ("mix.right.v", r.out_rows))
        silu = at
        put("gate", ("mix.right.g", r.out_rows))
        put("attention", ("mix.left.q", l.q_rows), ("mix.left.k", l.k_rows), ("mix.left.v", l.v_rows))
        at = plain = exact = round_up(at, BLOCK_COLUMNS)
    else:
        put("recurrence", ("mix.q", m.heads * m.dim), ("mix.k", m.heads * m.dim), ("mix.v", m.out_rows))
        put("gate", ("mix.g", m.out_rows))
        at = plain = round_up(at, BLOCK_COLUMNS)
        put("logits", ("mix.i", m.heads), ("mix.f", m.heads))
        at = exact = round_up(at, BLOCK_COLUMNS)
    parts["ff"] = at
    ff = f.ff if f is not None else 0
    return BlockLayout(parts, tuple(src), silu, plain, exact, at + 2 * ff, at + ff)


@dataclass(frozen=True)
class LayeredSpec:
    """A decoder whose layers are listed one by one: an fp32 residual stream, layers of unequal kinds and sizes, a looped range.
    A *run* is one execution of a layer; every run has its own cache or state.  ``block``: "sandwich" (a norm before and after each
    sublayer) or "parallel" (mixer and feed-forward read one layer norm and are added together; the head is the embedding table)."""
    name: str
    arch: str
    hidden: int
    vocab: int
    layers: tuple
    eps: float = 1e-6
    loop: LoopSpec | None = None
    seed: int = 20240531
    bits: int = 16
    block: str = "sandwich"
    logit_scale: float = 1.0

    def __post_init__(self):
        lp = self.loop
        if self.block not in ("sandwich", "parallel") or not self.layers or self.hidden < 1 or self.vocab < 1:
            raise ValueError(f"{self.name}: block {self.block!r}, {len(self.layers)} layers, width {self.hidden}, vocabulary {self.vocab}")
        if lp is not None and not (self.block == "sandwich" and 0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError(f"{self.name}: loop {lp} does not fit {len(self.layers)} layers")
        mixers, ffs = ((AttentionSpec,), MoeSpec) if self.block == "sandwich" else ((ParallelMixerSpec, MatrixMemorySpec), ClampedGluSpec)
        for i, l in enumerate(self.layers):
            m, f = l.mixer, l.mlp
            if not isinstance(m, mixers) or not m.check():
                raise ValueError(f"{self.name}: layer {i}: attention sizes {m}" if isinstance(m, AttentionSpec) else f"{self.name}: layer {i}: mixer sizes {m}")
            if f is not None and not (isinstance(f, ffs) and f.check()):
                raise ValueError(f"{self.name}: layer {i}: expert sizes {f}" if isinstance(f, MoeSpec) else f"{self.name}: layer {i}: feed-forward sizes {f}")

    def runs(self) -> list:
        """(layer, the embedding output is added first) in execution order."""
        lp, n = self.loop, len(self.layers)
        if lp is None:
            return [(i, False) for i in range(n)]
        body = [(i, k > 0 and i == lp.start) for k in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, False) for i in range(lp.start)] + body + [(i, False) for i in range(lp.stop, n)]

    @property
    def recurrent(self) -> bool:
        """Some layer carries a state that summarises all positions before: a sequence can only be continued, not rewound."""
        return self.block == "parallel"

    def _attention(self):
        """The softmax attention of every run that has one."""
        for i, _ in self.runs():
            m = self.layers[i].mixer
            if isinstance(m, (AttentionSpec, ParallelMixerSpec)):
                yield m.left if isinstance(m, ParallelMixerSpec) else m

    def _recurrences(self):
        for i, _ in self.runs():
            m = self.layers[i].mixer
            if not isinstance(m, AttentionSpec):
                yield m.right if isinstance(m, ParallelMixerSpec) else m

    # ---- algorithmic bytes of a decode step at bf16: every weight that is used once, the keys and values, the states
    def weight_bytes_per_token(self) -> int:
        tot, D = self.hidden * self.vocab, self.hidden
        for i, _ in self.runs():
            m, f = self.layers[i].mixer, self.layers[i].mlp
            if self.block == "parallel":
                tot += D * (sum(n for _, _, n in block_layout(self.layers[i]).sources) + (3 * f.ff if f is not None else 0))
                tot += D * (m.left.out_rows + m.right.out_rows if isinstance(m, ParallelMixerSpec) else m.out_rows)
                continue
            tot += m.rows * D + D * m.heads * m.vdim
            if f is not None:
                tot += D * (f.experts + 2 * f.shared_ff + 2 * f.top * f.ff)
        return 2 * tot

    def kv_bytes_per_token(self, ctx: int) -> int:
        return (sum(2 * m.visible(ctx) * (m.k_rows + m.v_rows) for m in self._attention())
                + sum(8 * m.heads * m.dim * m.vdim for m in self._recurrences()))            # a state is fp32, read and written

    def bytes_per_token(self, ctx: int) -> int:
        return self.weight_bytes_per_token() + self.kv_bytes_per_token(ctx)

    def flops_per_token(self, ctx: float) -> float:
        """Multiply-adds x 2 of one position that sees ``ctx`` keys, the head left out (prompt positions need no logits)."""
        w = self.weight_bytes_per_token() // 2 - self.hidden * self.vocab
        att = sum(m.heads * m.maps * (m.dim + m.vdim) * m.visible(int(ctx)) for m in self._attention())
        return 2.0 * (w + att + sum(2 * m.heads * m.dim * m.vdim for m in self._recurrences()))


def _fatulix(name, hidden, vocab, n_layers, attn, mlp, loop=None):
    return LayeredSpec(name, "Fatulix", hidden, vocab, tuple(LayerSpec(attn, mlp) for _ in range(n_layers)), loop=loop)


def _kakunex(name, hidden, vocab, order, left, right, memory, mlp, logit_scale=1.0):
    """``order``: "p" for a layer with the parallel mixer, "m" for one with the matrix memory."""
    mix = {"p": ParallelMixerSpec(left, right), "m": memory}
    return LayeredSpec(name, "Kakunex", hidden, vocab, tuple(LayerSpec(mix[c], mlp) for c in order), eps=1e-5, block="parallel", logit_scale=logit_scale)


def _kakunex_left(heads, kv_heads, window, keep):
    """Rotary windowed attention of head size 128."""
    return AttentionSpec(heads, kv_heads, 128, 128, 128 ** -0.5, norm="projection", gate=False, rotary=RotarySpec(128, 5e5, FrequencyScaling(8.0, 1.0, 4.0, 8192)),
                         window=window, keep_first=keep)


def _slopes(n):
    """Decays of n heads, from fast to slow."""
    return tuple(math.exp(-2.0 ** (-8.0 * (i + 1) / n)) for i in range(n))


CONFIGS = {
    # Qwen2.5-0.5B-shaped (CPU-reference-sized parity config)
    "qwen2.5-0.5b": ModelSpec("qwen2.5-0.5b", "qwen2", 24, 896, 14, 2, 64, 4864, 151936),
    # Qwen2.5-7B-shaped (headline metric)
    "qwen2.5-7b": ModelSpec("qwen2.5-7b", "qwen2", 28, 3584, 28, 4, 128, 18944, 152064),
    # Gemma-3-4B-shaped: GeGLU-tanh, sliding window 1024 on 5 of every 6 layers
    "gemma3-4b": ModelSpec("gemma3-4b", "gemma3", 34, 2560, 8, 4, 256, 10240, 262144, window=1024, global_every=6),
    # Qwen2.5-32B-shaped (tensor-parallel config)
    "qwen2.5-32b": ModelSpec("qwen2.5-32b", "qwen2", 64, 5120, 40, 8, 128, 27648, 152064),
    # tiny shapes for fast parity tests (not benchmark configs)
    "tiny-qwen": ModelSpec("tiny-qwen", "qwen2", 2, 256, 4, 2, 64, 512, 1024),
    "tiny-gemma": ModelSpec("tiny-gemma", "gemma3", 3, 256, 4, 2, 64, 512, 1024, window=16, global_every=3),
}


LAYERED_CONFIGS = {
    # looped mixture-of-experts decoders with differential attention, at sizes of the layers of a small, a 7B and a 32B model
    "fatulix-2048": _fatulix("fatulix-2048", 2048, 65536, 16, AttentionSpec(16, 4, 64, 128, 0.125, 0.3), MoeSpec(32, 4, 1024, 2048), LoopSpec(4, 8, 2)),
    "fatulix-3584": _fatulix("fatulix-3584", 3584, 152064, 8, AttentionSpec(28, 4, 64, 128, 0.125, 0.3), MoeSpec(16, 2, 4672, 9344)),
    "fatulix-5120": _fatulix("fatulix-5120", 5120, 152064, 6, AttentionSpec(40, 8, 64, 128, 0.125, 0.3), MoeSpec(8, 2, 8192, 8192)),
    "tiny-fatulix": _fatulix("tiny-fatulix", 128, 320, 3, AttentionSpec(6, 2, 24, 32, 0.2, 0.4), MoeSpec(5, 2, 64, 128), LoopSpec(1, 3, 2)),
    # parallel blocks of windowed attention beside linear attention, with matrix-memory layers between, at the widths above
    "kakunex-2048": _kakunex("kakunex-2048", 2048, 65536, "pppmpppm" * 2, _kakunex_left(16, 4, 1024, 64), LightningSpec(16, 128, 128, _slopes(16)),
                             MatrixMemorySpec(8, 128, 256, 15.0), ClampedGluSpec(4096, 7.0)),
    "kakunex-3584": _kakunex("kakunex-3584", 3584, 152064, "pppmpppm", _kakunex_left(28, 4, 1024, 64), LightningSpec(28, 128, 128, _slopes(28)),
                             MatrixMemorySpec(14, 128, 256, 15.0), ClampedGluSpec(12416, 7.0)),
    "kakunex-5120": _kakunex("kakunex-5120", 5120, 152064, "ppmppm", _kakunex_left(40, 8, 1024, 64), LightningSpec(40, 128, 128, _slopes(40)),
                             MatrixMemorySpec(20, 128, 256, 15.0), ClampedGluSpec(16384, 7.0)),
    "tiny-kakunex": _kakunex("tiny-kakunex", 128, 352, "pmp",
                             AttentionSpec(4, 2, 32, 16, 0.2, norm="projection", gate=False, rotary=RotarySpec(24, 1e4, FrequencyScaling(2.0, 1.0, 3.0, 64)), window=24, keep_first=3),
                             LightningSpec(4, 16, 16, (0.5, 0.8, 0.95, 1.0)), MatrixMemorySpec(2, 24, 32, 10.0), ClampedGluSpec(192, 2.0), 1.5),
}


def config(name: str):
    """The registered shape called ``name``: a ModelSpec or a LayeredSpec."""
    if name in CONFIGS:
        return CONFIGS[name]
    if name in LAYERED_CONFIGS:
        return LAYERED_CONFIGS[name]
    raise KeyError(f"no configuration {name!r}; known: {sorted(CONFIGS) + sorted(LAYERED_CONFIGS)}")


# ---- tensor naming / stream ids (FNV-1a 64 of the name, xor a mix of the seed) ----
def _mix64(z: int) -> int:
    z = (z + 0x9E3779B97F4A7C15) & MASK64
    z = ((z ^ (z >> 30)) * 0xBF58476D1CE4E5B9) & MASK64
    z = ((z ^ (z >> 27)) * 0x94D049BB133111EB) & MASK64
    return z ^ (z >> 31)


def stream_id(seed: int, name: str) -> int:
    h = 0xCBF29CE484222325
    for b in name.encode():
        h = ((h ^ b) * 0x100000001B3) & MASK64
    return h ^ _mix64(seed)


def tensor_name(layer: int, leaf: str) -> str:
    return leaf if layer < 0 else f"layers.{layer}.{leaf}"
