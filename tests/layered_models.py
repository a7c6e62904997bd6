"""Small layered decoders with random weights for the tests, handed to the engine and to the plain oracle alike."""
from __future__ import annotations

import numpy as np

from fusekit_b200 import checkpoint as CK
from fusekit_b200.layered import LayeredEngine, tensor_shapes
from fusekit_b200.model_spec import (AttentionSpec, ClampedGluSpec, FrequencyScaling, LayeredSpec, LayerSpec, LightningSpec, LoopSpec, MatrixMemorySpec, MoeSpec,
                                     ParallelMixerSpec, RotarySpec)
from oracle.layered import LayeredOracle, ParallelBlockOracle


def bits(a):
    return CK.f32_to_bf16_bits(np.asarray(a, np.float32))


def values(b):
    return (np.asarray(b, np.uint16).astype(np.uint32) << 16).view(np.float32)


def rounded(a):
    """float32 values that bf16 holds exactly."""
    return values(bits(a))


def spec(layers, hidden=96, vocab=211, loop=None, eps=1e-5, name="test"):
    return LayeredSpec(name, "Fatulix", hidden, vocab, tuple(layers), eps=eps, loop=loop)


def random_tensors(s, seed=0, router=6.0):
    """name -> bf16 bits.  Norm weights vary around 1, q/k norm weights are large enough for peaked attention, and the router is
    scaled so that its choices are rarely close."""
    rng = np.random.default_rng(seed)
    t = {}
    for n, shape in sorted(tensor_shapes(s).items()):
        a = rng.standard_normal(shape)
        if n == "embed":
            a *= 1.0
        elif n.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            a *= 0.25
        elif n.endswith(("q.norm", "k.norm")):
            a = 1.3 + 0.3 * a
        elif n.endswith(".f.b"):
            a = 3.0 + a                                  # long memories
        elif n.endswith(".b"):
            a *= 0.5
        elif len(shape) == 1:
            a = 1.0 + 0.2 * a
        else:
            a *= shape[1] ** -0.5 * (router if n.endswith("router") else 1.0)
        t[n] = bits(a)
    return t


def engine(s, tensors, capacity, dtype="float32", **kw):
    e = LayeredEngine(s, capacity, dtype=dtype, **kw)

    def prov(name, shape):
        assert tensors[name].shape == tuple(shape), name
        return tensors[name]
    e.load_from(prov)
    return e


def oracle(s, tensors):
    return (ParallelBlockOracle if s.block == "parallel" else LayeredOracle)(s, {k: values(v) for k, v in tensors.items()})


def parallel_entry(m, f):
    if isinstance(m, ParallelMixerSpec):
        l, r, rot = m.left, m.right, m.left.rotary
        left = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale,
                "mask": None if l.window is None else {"size": l.window, "keep_first": l.keep_first},
                "rot": None if rot is None else {"dims": rot.dims, "base": rot.base, "scaling": None if rot.scaling is None else vars(rot.scaling)}}
        e = {"type": "parallel", "mixer": {"left": left, "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)}}}
    else:
        e = {"type": "mlstm", "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}}
    e["mlp"] = None if f is None else {"kind": "dense", "ff": f.ff, "limit": f.limit}
    return e


def write_model(path, s, tensors):
    """A model directory as the loader reads it."""
    import json
    import os
    os.makedirs(path, exist_ok=True)
    layers = []
    for l in s.layers:
        m, f = l.mixer, l.mlp
        if s.block == "parallel":
            layers.append(parallel_entry(m, f))
            continue
        layers.append({"type": "attention", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff},
                       "mlp": None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff},
                                                      "shared": {"ff": f.shared_ff} if f.shared_ff else None}})
    cfg = {"architecture": s.arch, "width": s.hidden, "vocab": s.vocab, "norm": {"eps": s.eps}, "layers": layers}
    if s.block == "parallel":
        cfg["logit_scale"] = s.logit_scale
    if s.loop is not None:
        cfg["loop"] = {"start": s.loop.start, "stop": s.loop.stop, "times": s.loop.times}
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    CK.write_safetensors(os.path.join(path, "model.safetensors"), {k: (v, "BF16") for k, v in tensors.items()})


A, M = AttentionSpec, MoeSpec
# shapes that differ layer by layer, sizes off every tile (8, 16, 64), grouped and ungrouped heads, one expert chosen and all
# chosen, a layer without feed-forward, a feed-forward without shared expert, a loop that starts late / runs three times
SPECS = {
    "mixed": spec([LayerSpec(A(4, 2, 24, 40, 0.31, 0.2), M(7, 3, 40, 56)), LayerSpec(A(6, 6, 8, 20, 0.5, 0.45), None),
                   LayerSpec(A(3, 1, 36, 28, 0.25, 0.7), M(4, 4, 24, 0)), LayerSpec(A(5, 1, 16, 72, 0.35, 0.1), M(9, 1, 100, 33))],
                  hidden=88, loop=LoopSpec(1, 3, 3)),
    "wide-heads": spec([LayerSpec(A(4, 4, 72, 136, 0.12, 0.35), M(6, 2, 64, 64)), LayerSpec(A(2, 1, 128, 200, 0.09, 0.5), M(3, 2, 130, 70))], hidden=130, vocab=301,
                       loop=LoopSpec(0, 1, 2)),
    "many-rows": spec([LayerSpec(A(10, 1, 20, 16, 0.3, 0.25), M(70, 5, 16, 24)), LayerSpec(A(12, 3, 64, 64, 0.15, 0.6), M(33, 6, 72, 8))], hidden=200, vocab=97),
    "plain-maps": spec([LayerSpec(A(4, 2, 48, 64, 0.2, None), M(8, 2, 64, 96))], hidden=128, vocab=130),
    "one-layer": spec([LayerSpec(A(1, 1, 8, 8, 0.6, 0.3), M(1, 1, 8, 8))], hidden=16, vocab=33, loop=LoopSpec(0, 1, 1)),
}


def parallel_spec(layers, hidden=96, vocab=211, eps=1e-5, logit_scale=1.0, name="test"):
    return LayeredSpec(name, "Kakunex", hidden, vocab, tuple(layers), eps=eps, block="parallel", logit_scale=logit_scale)


def windowed(heads, kv_heads, dim, vdim, scale, window=None, keep=0, rot=None, scaling=None, base=1e4):
    r = None if rot is None else RotarySpec(rot, base, None if scaling is None else FrequencyScaling(*scaling))
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, norm="projection", gate=False, rotary=r, window=window, keep_first=keep)


P, L, MM, G = ParallelMixerSpec, LightningSpec, MatrixMemorySpec, ClampedGluSpec
# sizes off every tile, unequal layers, windows of one / none / larger than a tile, no kept keys / more than a tile of them, rotation of all / some / no
# dimensions, with and without stretching, decays of 0 and 1, layers without feed-forward, widths that no vector load fits
PARALLEL_SPECS = {
    "mixed": parallel_spec([LayerSpec(P(windowed(4, 2, 24, 40, 0.3, 20, 5, 16, (4.0, 1.0, 4.0, 50.0)), L(3, 16, 24, (0.5, 0.9, 1.0))), G(72, 0.8)),
                            LayerSpec(MM(3, 24, 40, 8.0), None), LayerSpec(P(windowed(3, 1, 20, 12, 0.25, 1, 0, 20), L(1, 40, 72, (0.97,))), None),
                            LayerSpec(MM(1, 8, 136, 20.0), G(40, 3.0)), LayerSpec(P(windowed(5, 5, 8, 16, 0.5, None, 0, None), L(5, 8, 8, (0.0, 0.3, 0.6, 0.8, 0.999))), G(24, 100.0))],
                           hidden=88, logit_scale=1.7),
    "memory-first": parallel_spec([LayerSpec(MM(2, 72, 16, 5.0), G(136, 1.0)), LayerSpec(MM(4, 16, 64, 15.0), G(8, 0.5)),
                                   LayerSpec(P(windowed(2, 2, 40, 64, 0.2, 70, 66, 40, (8.0, 1.0, 2.0, 30.0)), L(2, 136, 64, (0.99, 0.8))), G(64, 2.0))], hidden=136, vocab=130),
    "odd-sizes": parallel_spec([LayerSpec(P(windowed(6, 3, 18, 22, 0.25, 33, 3, 6, (2.0, 1.0, 3.0, 40.0)), L(3, 10, 14, (0.7, 0.95, 0.2))), G(37, 1.2)),
                                LayerSpec(MM(3, 14, 18, 11.0), G(21, 0.9)), LayerSpec(MM(2, 5, 7, 6.0), None)], hidden=75, vocab=99, eps=1e-3, logit_scale=0.4),
    "wide-heads": parallel_spec([LayerSpec(P(windowed(12, 1, 136, 200, 0.1, 40, 10, 136), L(1, 264, 130, (0.9,))), G(48, 4.0)),
                                 LayerSpec(MM(1, 200, 72, 15.0), G(33, 2.0))], hidden=64, vocab=80),
    "memory-only": parallel_spec([LayerSpec(MM(2, 12, 20, 6.0), None)], hidden=36, vocab=50),
    "one-layer": parallel_spec([LayerSpec(P(windowed(1, 1, 8, 8, 0.6, 4, 2, 8), L(1, 8, 8, (0.9,))), G(8, 1.0))], hidden=16, vocab=33, logit_scale=3.0),
}


def logit_error(got, want):
    """Root mean square over the vocabulary of the difference (means taken off), per row, over the reference's spread."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2))
