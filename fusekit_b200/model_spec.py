"""Decoder shapes of the benchmark configs and the naming of their seeded tensors.

The reference learns these from ``config.json`` (``ModelMeta::from_config_file``,
src/fusion/ir.rs:604-749) and from the traced graph; capture needs MLX, so the five
benchmark shapes are stated here directly.
"""
from __future__ import annotations

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
class AttentionSpec:
    """Attention with an RMS norm on every q/k (sub-)head, no rotation and a sigmoid output gate per head.  ``diff`` set:
    differential attention -- every head has two query/key maps over the same values, combined as a1 - lambda a2."""
    heads: int
    kv_heads: int
    dim: int                  # query/key size of a map
    vdim: int
    scale: float              # score = (q . k) * scale
    diff: float | None = None

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
        return self.q_rows + self.k_rows + self.v_rows + self.heads


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of ``experts`` feed-forward layers W_down relu(W_up h)^2, ``top`` per token weighted by the softmax over the
    chosen router logits, plus a shared one of size ``shared_ff`` (0: none)."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: MoeSpec | None = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row; the embedding output is added to x before each repetition."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayeredSpec:
    """A decoder whose layers are listed one by one: norms before and after each sublayer, an fp32 residual stream, layers of
    unequal sizes, a looped range.  A *run* is one execution of a layer; every run has its own cache."""
    name: str
    arch: str
    hidden: int
    vocab: int
    layers: tuple
    eps: float = 1e-6
    loop: LoopSpec | None = None
    seed: int = 20240531
    bits: int = 16

    def __post_init__(self):
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError(f"{self.name}: loop {lp} does not fit {len(self.layers)} layers")
        for i, l in enumerate(self.layers):
            m, f = l.mixer, l.mlp
            if min(m.heads, m.kv_heads, m.dim, m.vdim) < 1 or m.heads % m.kv_heads:
                raise ValueError(f"{self.name}: layer {i}: attention sizes {m}")
            if f is not None and not (1 <= f.top <= f.experts and f.ff >= 1 and f.shared_ff >= 0):
                raise ValueError(f"{self.name}: layer {i}: expert sizes {f}")

    def runs(self) -> list:
        """(layer, the embedding output is added first) in execution order."""
        lp, n = self.loop, len(self.layers)
        if lp is None:
            return [(i, False) for i in range(n)]
        body = [(i, k > 0 and i == lp.start) for k in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, False) for i in range(lp.start)] + body + [(i, False) for i in range(lp.stop, n)]

    # ---- algorithmic bytes of a decode step at bf16: every weight that is used once, and the keys and values
    def weight_bytes_per_token(self) -> int:
        tot = self.hidden * self.vocab
        for i, _ in self.runs():
            m, f = self.layers[i].mixer, self.layers[i].mlp
            tot += m.rows * self.hidden + self.hidden * m.heads * m.vdim
            if f is not None:
                tot += self.hidden * (f.experts + 2 * f.shared_ff + 2 * f.top * f.ff)
        return 2 * tot

    def kv_bytes_per_token(self, ctx: int) -> int:
        return sum(2 * ctx * (self.layers[i].mixer.k_rows + self.layers[i].mixer.v_rows) for i, _ in self.runs())

    def bytes_per_token(self, ctx: int) -> int:
        return self.weight_bytes_per_token() + self.kv_bytes_per_token(ctx)

    def flops_per_token(self, ctx: float) -> float:
        """Multiply-adds x 2 of one position that sees ``ctx`` keys, the head left out (prompt positions need no logits)."""
        w = self.weight_bytes_per_token() // 2 - self.hidden * self.vocab
        att = sum(self.layers[i].mixer.heads * self.layers[i].mixer.maps * (self.layers[i].mixer.dim + self.layers[i].mixer.vdim) for i, _ in self.runs())
        return 2.0 * (w + att * ctx)


def _fatulix(name, hidden, vocab, n_layers, attn, mlp, loop=None):
    return LayeredSpec(name, "Fatulix", hidden, vocab, tuple(LayerSpec(attn, mlp) for _ in range(n_layers)), loop=loop)


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
