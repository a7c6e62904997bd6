"""Small layered decoders with random weights for the tests, handed to the engine and to the plain oracle alike."""
from __future__ import annotations

import numpy as np

from fusekit_b200 import checkpoint as CK
from fusekit_b200.layered import LayeredEngine, tensor_shapes
from fusekit_b200.model_spec import AttentionSpec, LayeredSpec, LayerSpec, LoopSpec, MoeSpec
from oracle.layered import LayeredOracle


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
    return LayeredOracle(s, {k: values(v) for k, v in tensors.items()})


def write_model(path, s, tensors):
    """A model directory as the loader reads it."""
    import json
    import os
    os.makedirs(path, exist_ok=True)
    layers = []
    for l in s.layers:
        m, f = l.mixer, l.mlp
        layers.append({"type": "attention", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff},
                       "mlp": None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff},
                                                      "shared": {"ff": f.shared_ff} if f.shared_ff else None}})
    cfg = {"architecture": s.arch, "width": s.hidden, "vocab": s.vocab, "norm": {"eps": s.eps}, "layers": layers}
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


def logit_error(got, want):
    """Root mean square over the vocabulary of the difference (means taken off), per row, over the reference's spread."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2))
