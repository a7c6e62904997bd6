"""Layered decoders, host side: configuration, registry, plans, task graphs and the plain oracle's own consistency."""
import ctypes as C
import json

import numpy as np
import pytest

from fusekit_b200 import _native as N
from fusekit_b200 import checkpoint as CK
from fusekit_b200 import config
from fusekit_b200 import task_graph as TG
from fusekit_b200.layered import combination_constant, rotation_table, weight_plan
from fusekit_b200.model_spec import LAYERED_CONFIGS, LayeredSpec, LoopSpec, block_layout
from oracle import layered as OL
from tests import layered_models as LM


@pytest.mark.parametrize("name", sorted(LM.SPECS))
def test_configuration_round_trip(tmp_path, name):
    s = LM.SPECS[name]
    if any(l.mixer.diff is None for l in s.layers):
        pytest.skip("the file format always names the combination constant")
    t = LM.random_tensors(s)
    LM.write_model(tmp_path / "m", s, t)
    ck = CK.LayeredCheckpoint(str(tmp_path / "m"))
    try:
        got = ck.spec
        assert (got.layers, got.loop, got.hidden, got.vocab, got.eps) == (s.layers, s.loop, s.hidden, s.vocab, s.eps)
        prov = ck.provider()
        for n, shape in LM.tensor_shapes(s).items():
            assert np.array_equal(prov(n, shape), t[n])
        with pytest.raises(ValueError, match="shape"):
            prov("embed", (1, 1))
        with pytest.raises(KeyError):
            prov("l9.nothing", (1,))
    finally:
        ck.close()


@pytest.mark.parametrize("name", sorted(LM.PARALLEL_SPECS))
def test_parallel_configuration_round_trip(tmp_path, name):
    s = LM.PARALLEL_SPECS[name]
    t = LM.random_tensors(s)
    LM.write_model(tmp_path / "m", s, t)
    ck = CK.LayeredCheckpoint(str(tmp_path / "m"))
    try:
        got = ck.spec
        assert (got.layers, got.block, got.hidden, got.vocab, got.eps, got.logit_scale) == (s.layers, "parallel", s.hidden, s.vocab, s.eps, s.logit_scale)
        for n, shape in LM.tensor_shapes(s).items():
            assert np.array_equal(ck.provider()(n, shape), t[n])
    finally:
        ck.close()
    cfg = json.load(open(tmp_path / "m" / "config.json"))
    for edit, what in ((lambda c: c["layers"][0].update(type="scan"), "mixer type"), (lambda c: c["layers"][0].update(mlp={"kind": "moe"}), "feed-forward kind")):
        c = json.loads(json.dumps(cfg)); edit(c)
        with pytest.raises(ValueError, match=what):
            CK.layered_spec_from_config(c)


def test_parallel_sizes_are_checked():
    w, l = LM.windowed(4, 2, 8, 8, 0.3, 5), LM.L(2, 8, 8, (0.5, 0.9))
    for m in (LM.P(LM.windowed(4, 3, 8, 8, 0.3, 5), l), LM.P(LM.windowed(4, 2, 8, 8, 0.3, 0), l), LM.P(LM.windowed(4, 2, 8, 8, 0.3, 5, rot=10), l),
              LM.P(LM.windowed(4, 2, 8, 8, 0.3, 5, rot=3), l), LM.P(w, LM.L(2, 8, 8, (0.5,))), LM.P(w, LM.L(1, 8, 8, (1.5,))), LM.MM(2, 8, 8, 0.0), LM.A(2, 1, 8, 8, 0.5, 0.3)):
        with pytest.raises(ValueError, match="sizes"):
            LM.parallel_spec([LM.LayerSpec(m, None)])
    with pytest.raises(ValueError, match="feed-forward"):
        LM.parallel_spec([LM.LayerSpec(LM.P(w, l), LM.G(8, 0.0))])
    with pytest.raises(ValueError, match="mixer"):
        LM.spec([LM.LayerSpec(LM.P(w, l), None)])


def test_unknown_mechanisms_are_refused_by_name(tmp_path):
    s = LM.SPECS["mixed"]
    LM.write_model(tmp_path / "m", s, LM.random_tensors(s))
    cfg = json.load(open(tmp_path / "m" / "config.json"))
    for edit, what in ((lambda c: c.update(architecture="Other"), "architecture"), (lambda c: c["layers"][0].update(type="scan"), "mixer type"),
                       (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"), (lambda c: c.update(loop={"start": 3, "stop": 9, "times": 2}), "loop"),
                       (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "attention sizes")):
        c = json.loads(json.dumps(cfg)); edit(c)
        with pytest.raises(ValueError, match=what):
            CK.layered_spec_from_config(c)


def test_runs_of_a_looped_model():
    s = LM.SPECS["mixed"]
    assert s.runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert LM.SPECS["wide-heads"].runs() == [(0, False), (0, True), (1, False)]
    assert LM.SPECS["one-layer"].runs() == [(0, False)]
    with pytest.raises(ValueError):
        LayeredSpec("x", "Fatulix", 8, 8, s.layers, loop=LoopSpec(2, 2, 2))


def test_registry_knows_the_layered_shapes():
    for n in LAYERED_CONFIGS:
        assert config(n) is LAYERED_CONFIGS[n]
    assert config("qwen2.5-7b").hidden == 3584
    with pytest.raises(KeyError):
        config("nothing")
    s = LAYERED_CONFIGS["fatulix-2048"]
    m, f = s.layers[0].mixer, s.layers[0].mlp
    per_run = m.rows * 2048 + 2048 * m.heads * m.vdim + 2048 * (f.experts + 2 * f.shared_ff + 2 * f.top * f.ff)
    assert s.weight_bytes_per_token() == 2 * (len(s.runs()) * per_run + 2048 * s.vocab)


@pytest.mark.parametrize("name", sorted(LM.SPECS))
def test_decode_graph_round_trips_through_the_library(name):
    """Every role of the graph is one the engine resolves, and the library's own reader rebuilds the same records."""
    s = LM.SPECS[name]
    g = json.loads(json.dumps(TG.emit_layered(s, 100, {i: 0.1 * i for i in range(len(s.layers))}, dtype=1)))
    runs = s.runs()
    kinds = [t["kind"] for t in g["tasks"]]
    assert kinds.count(TG.K_ATTDEC) == len(runs) and kinds[0] == TG.K_EMBEDROWS and kinds[-1] == TG.K_NORMLIN
    assert kinds.count(TG.K_MOEDOWN) == sum(s.layers[i].mlp is not None for i, _ in runs)
    adds = [t["layer_idx"] for t in g["tasks"] if t["kind"] == TG.K_NORMLIN and 3 in TG.task_slots(t)]
    assert adds == [r for r, (_, again) in enumerate(runs) if again]
    caches = {TG.task_slots(t)[3] for t in g["tasks"] if t["kind"] == TG.K_ATTDEC}
    assert len(caches) == len(runs)                       # every pass has a cache of its own
    roles = sorted({b["role"] for t in g["tasks"] for b in t["extra_bindings"] if b["slot"] < 100})
    table = (N.RoleBinding * len(roles))(*[N.RoleBinding(r.encode(), 4096 + i) for i, r in enumerate(roles)])
    n, out = C.c_int32(), (N.Task * len(kinds))()
    N.check(N.lib().fk_tasks_from_json(json.dumps(g).encode(), table, len(roles), out, len(kinds), C.byref(n)))
    assert n.value == len(kinds)
    for got, t in zip(out, g["tasks"]):
        assert got.kind == t["kind"] and list(got.iarg)[:len(t["iargs"])] == t["iargs"]
        assert np.allclose(list(got.farg)[:len(t["fargs"])], t["fargs"], rtol=1e-6)


def test_weight_plan_covers_every_matrix_once():
    s = LM.SPECS["many-rows"]
    names = [n for _, parts, _ in weight_plan(s) for n, _ in parts]
    assert len(names) == len(set(names)) == 1 + sum(4 + 1 + 1 + 2 * l.mlp.experts + 2 for l in s.layers)


@pytest.mark.parametrize("name", sorted(LM.PARALLEL_SPECS))
def test_parallel_decode_graph_round_trips_through_the_library(name):
    s = LM.PARALLEL_SPECS[name]
    g = json.loads(json.dumps(TG.emit_layered(s, 100, {}, dtype=1)))
    kinds = [t["kind"] for t in g["tasks"]]
    both = sum(isinstance(l.mixer, LM.P) for l in s.layers)
    assert kinds.count(TG.K_WINDEC) == both and kinds.count(TG.K_RECDEC) == kinds.count(TG.K_SEGLIN) == len(s.layers) and len(kinds) == 2 + 3 * len(s.layers) + both
    states = {TG.task_slots(t)[6] for t in g["tasks"] if t["kind"] == TG.K_RECDEC}
    assert len(states) == len(s.layers)
    roles = sorted({b["role"] for t in g["tasks"] for b in t["extra_bindings"] if b["slot"] < 100})
    table = (N.RoleBinding * len(roles))(*[N.RoleBinding(r.encode(), 4096 + i) for i, r in enumerate(roles)])
    n, out = C.c_int32(), (N.Task * len(kinds))()
    N.check(N.lib().fk_tasks_from_json(json.dumps(g).encode(), table, len(roles), out, len(kinds), C.byref(n)))
    assert n.value == len(kinds)
    for got, t in zip(out, g["tasks"]):
        assert got.kind == t["kind"] and list(got.iarg)[:len(t["iargs"])] == t["iargs"]
        assert np.allclose(list(got.farg)[:len(t["fargs"])], t["fargs"], rtol=1e-6)


@pytest.mark.parametrize("name", sorted(LM.PARALLEL_SPECS))
def test_block_layout_places_every_tensor_once(name):
    s = LM.PARALLEL_SPECS[name]
    for i, l in enumerate(s.layers):
        b = block_layout(l)
        assert b.plain % 32 == 0 and b.exact % 32 == 0 and 0 <= b.silu <= b.plain <= b.exact <= b.rows
        rows = np.zeros(b.exact, int)
        for _, at, n in b.sources:
            rows[at:at + n] += 1
        assert rows.max() == 1 and b.rows - b.exact == (2 * l.mlp.ff if l.mlp else 0) == 2 * (b.out_rows - b.exact)
        for leaf, at, n in b.sources:                     # the logits of the gates are kept apart, silu covers the linear attention's q, k, v
            assert (at >= b.plain) == (leaf in ("mix.i", "mix.f"))
            assert (at < b.silu) == leaf.startswith(("mix.right.q", "mix.right.k", "mix.right.v"))
        parts = {p: n for p, n, _ in weight_plan(s)}[f"layer_param.{i}.block"]
        assert sum(n for _, n in parts) == b.rows
    names = [t for _, parts, _ in weight_plan(s) for n, _ in parts if n for t in (n if isinstance(n, tuple) else (n,))]
    assert len(names) == len(set(names))


def test_visible_keys_counts():
    w = LM.windowed(1, 1, 8, 8, 1.0, 5, 3)
    for ctx in range(1, 30):
        p = ctx - 1
        assert w.visible(ctx) == sum(p - j < 5 or j < 3 for j in range(ctx))
    assert LM.windowed(1, 1, 8, 8, 1.0).visible(77) == 77


def test_rotation_frequencies_match_the_oracle():
    for dims, base, sc in ((8, 1e4, None), (48, 3e5, (8.0, 1.0, 4.0, 300.0)), (64, 100.0, (3.0, 2.0, 2.5, 40.0)), (2, 5.0, (2.0, 1.0, 4.0, 7.0)), (0, 10.0, None)):
        r = LM.RotarySpec(dims, base, None if sc is None else LM.FrequencyScaling(*sc))
        assert np.allclose(r.frequencies(), OL.rotation_frequencies(dims, base, sc), rtol=1e-14)
        tab = rotation_table(r, 9)
        x = np.random.default_rng(dims).standard_normal((9, 1, dims + 3))
        want = OL.rotate_pairs(x, np.arange(9), OL.rotation_frequencies(dims, base, sc))
        u, v = x[:, 0, 0:dims:2], x[:, 0, 1:dims:2]
        assert np.allclose(u * tab[..., 0] - v * tab[..., 1], want[:, 0, 0:dims:2], atol=1e-6) and np.allclose(v * tab[..., 0] + u * tab[..., 1], want[:, 0, 1:dims:2], atol=1e-6)
        assert np.array_equal(want[..., dims:], x[..., dims:])
    f = OL.rotation_frequencies(16, 1e4, (4.0, 1.0, 4.0, 100.0)) / OL.rotation_frequencies(16, 1e4)
    assert f[0] == 1.0 and f[-1] == 0.25 and ((f > 0.25) & (f < 1.0)).any()       # all three ranges occur


def test_parallel_oracle_mechanisms_by_hand():
    assert np.allclose(OL.layer_norm(np.array([1.0, 3.0]), np.array([2.0, 2.0]), np.array([0.5, 0.0]), 3.0), [0.5 - 1.0, 1.0])
    g = OL.clamped_glu(np.array([5.0, -1.0]), np.array([-9.0, 0.5]), 2.0)
    assert np.allclose(g, [2.0 / (1 + np.exp(-3.404)) * -1.0, -1.0 / (1 + np.exp(1.702)) * 1.5])
    o, S = OL.decay_recurrence(np.ones((2, 1)), np.array([[2.0], [1.0]]), np.array([[1.0], [4.0]]), 0.5, np.zeros((1, 1)))
    assert np.allclose(o[:, 0], [2.0, 5.0]) and S[0, 0] == 5.0
    # one step from zero: m = max(f, i); the stored sums are scaled by exp(-m), which the floor of the divisor undoes
    o, (S, n, m) = OL.matrix_memory(np.array([[1.0]]), np.array([[0.5]]), np.array([[3.0]]), np.array([2.0]), np.array([-1.0]), (np.zeros((1, 1)), np.zeros(1), 0.0))
    assert m == 2.0 and np.allclose(S, 1.5) and np.allclose(o, 1.5 / (max(0.5, np.exp(-2)) + 1e-6))
    o, (S, n, m) = OL.matrix_memory(np.array([[0.01]]), np.array([[1.0]]), np.array([[1.0]]), np.array([-3.0]), np.array([-0.5]), (np.zeros((1, 1)), np.zeros(1), 0.0))
    assert m == -0.5 and np.allclose(o, 0.01 * np.exp(-2.5) / (np.exp(0.5) + 1e-6))
    v = np.arange(6.0)[:, None]                                                   # equal scores: the mean of what is seen
    got = OL.window_attention(np.zeros((6, 1)), np.zeros((6, 1)), v, 1.0, 0, 2, 1)[:, 0]
    assert np.allclose(got, [0, 0.5, 1.0, (0 + 2 + 3) / 3, (0 + 3 + 4) / 3, (0 + 4 + 5) / 3])
    assert np.allclose(OL.soft_cap(np.array([1e9, 0.001]), 4.0), [4.0, 0.001]) and np.allclose(OL.log_sigmoid(np.array([-800.0, 0.0])), [-800.0, -np.log(2)])


def test_parallel_oracle_does_not_depend_on_the_portions():
    s = LM.PARALLEL_SPECS["mixed"]
    t = LM.random_tensors(s, 3)
    toks = np.random.default_rng(1).integers(0, s.vocab, 40)
    whole = LM.oracle(s, t).forward(toks)
    for cuts in ([1] * 40, [2, 7, 31], [39, 1]):
        o, got, p = LM.oracle(s, t), [], 0
        for n in cuts:
            got.append(o.forward(toks[p:p + n])); p += n
        assert np.abs(np.concatenate(got) - whole).max() < 1e-9


def test_combination_constant():
    a, b, c, d = np.array([0.5, 1.0]), np.array([1.0, 0.25]), np.array([-1.0, 0.5]), np.array([0.5, 0.5])
    want = np.exp(0.75) - np.exp(-0.25) + 0.3
    assert abs(combination_constant(a, b, c, d, 0.3) - want) < 1e-12
    assert abs(OL.differential_lambda(a, b, c, d, 0.3) - want) < 1e-12


def test_oracle_does_not_depend_on_the_portions():
    s = LM.SPECS["mixed"]
    t = LM.random_tensors(s, 3)
    toks = np.random.default_rng(1).integers(0, s.vocab, 23)
    whole = LM.oracle(s, t).forward(toks)
    for cuts in ([1] * 23, [2, 7, 14], [22, 1]):
        o, got, p = LM.oracle(s, t), [], 0
        for n in cuts:
            got.append(o.forward(toks[p:p + n])); p += n
        assert np.abs(np.concatenate(got) - whole).max() < 1e-9


def test_oracle_mechanisms_by_hand():
    assert np.allclose(OL.rms(np.array([3.0, 4.0]), 0.0), np.array([3.0, 4.0]) / np.sqrt(12.5))
    assert np.allclose(OL.relu_squared(np.array([-2.0, 3.0])), [0.0, 9.0])
    idx, w = OL.route(np.array([[0.0, 2.0, 1.0, 2.0]]), 2)
    assert idx.tolist() == [[1, 3]] and np.allclose(w, 0.5)
    o = OL.differential_combine(np.array([1.0, 2.0]), np.array([1.0, 0.0]), 0.5, 0.2, 0.0)
    assert np.allclose(o, 0.8 * np.array([0.5, 2.0]) / np.sqrt((0.25 + 4.0) / 2))
    # two keys, the second one out of the first query's sight
    k, v = np.array([[1.0], [5.0]]), np.array([[1.0], [-1.0]])
    got = OL.softmax_attention(np.array([[1.0], [1.0]]), k, v, 1.0, 0)
    assert np.allclose(got[:, 0], [1.0, (np.exp(-4) - 1) / (np.exp(-4) + 1)])
