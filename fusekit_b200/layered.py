"""Engine of the layered decoders (``model_spec.LayeredSpec``): sandwiched sublayers (differential attention, mixture-of-experts
feed-forward, looped layers) or parallel blocks (windowed rotary attention beside linear attention, matrix memories, gated feed-forward).

It is a DecodeEngine in all but the layer: one position is a task graph captured as a CUDA graph and replayed with on-device
token feedback; several consecutive positions of a sequence (a prompt, or a portion of one) go through the row tasks.  Both
read and write the same caches, one per layer *run* -- a looped layer keeps keys and values for every pass, a recurrent mixer its
fp32 state.  A sequence owns a cache slot; closing it hands the slot to the next one, which overwrites the rows before it reads them
and does not read a state at position 0.  A sequence with a state can only be continued where it stands, or started again.

``dtype``: "bfloat16" keeps matrix-product operands and caches in bf16 (fp32 accumulation, fp32 residual, norms, scores and
router), "float32" keeps everything in fp32.  Weights are bf16 as stored in either case.
"""
from __future__ import annotations

import math

import numpy as np

from . import _native as N
from . import task_graph as TG
from .model_spec import AttentionSpec, LayeredSpec, ParallelMixerSpec, block_layout, stream_id
from .runtime import EngineBase, Runtime

MAX_ROWS = 2048          # positions per portion of a prompt


def weight_plan(spec: LayeredSpec) -> list:
    """(role, [(tensor, rows)], columns) of every matrix the kernels read: tensors stacked by rows; None for rows of zeros, a pair of
    tensors for their rows taken in turn."""
    D, out = spec.hidden, []
    for i, l in enumerate(spec.layers):
        m, f, p, t = l.mixer, l.mlp, f"layer_param.{i}.", f"l{i}."
        if spec.block == "parallel":
            lay, parts, at = block_layout(l), [], 0
            for leaf, row, n in lay.sources:
                parts += ([(None, row - at)] if row > at else []) + [(t + leaf, n)]
                at = row + n
            parts += [(None, lay.exact - at)] if lay.exact > at else []
            if f is not None:
                parts.append(((t + "mlp.gate", t + "mlp.up"), 2 * f.ff))
            out.append((p + "block", parts, D))
            for leaf, k in (("mix.left.o", m.left.out_rows), ("mix.right.o", m.right.out_rows)) if isinstance(m, ParallelMixerSpec) else (("mix.o", m.out_rows),):
                out.append((p + leaf, [(t + leaf, D)], k))
            if f is not None:
                out.append((p + "mlp.down", [(t + "mlp.down", D)], f.ff))
            continue
        out.append((p + "mix.qkvg", [(t + "mix.q", m.q_rows), (t + "mix.k", m.k_rows), (t + "mix.v", m.v_rows), (t + "mix.g", m.heads)], D))
        out.append((p + "mix.o", [(t + "mix.o", D)], m.heads * m.vdim))
        if f is None:
            continue
        out.append((p + "mlp.router_shared", [(t + "mlp.router", f.experts)] + ([(t + "mlp.shared.up", f.shared_ff)] if f.shared_ff else []), D))
        out.append((p + "mlp.experts_up", [(f"{t}mlp.e{e}.up", f.ff) for e in range(f.experts)], D))
        out.append((p + "mlp.experts_down", [(f"{t}mlp.e{e}.down", D) for e in range(f.experts)], f.ff))
        if f.shared_ff:
            out.append((p + "mlp.shared_down", [(t + "mlp.shared.down", D)], f.shared_ff))
    out.append(("param.lm_head", [("embed" if spec.block == "parallel" else "head", spec.vocab)], D))
    return out


def vector_plan(spec: LayeredSpec) -> list:
    """(role, tensor, shape, mean, std) of the embedding table, norm weights and biases (mean and std: synthetic values); several
    tensors of one shape lie one after the other."""
    D = spec.hidden
    if spec.block == "parallel":
        out = [("param.final_norm", "final.norm", (D,), 1.0, 0.02), ("param.final_norm.b", "final.norm.b", (D,), 0.0, 0.02)]
        for i, l in enumerate(spec.layers):
            m, p, t = l.mixer, f"layer_param.{i}.", f"l{i}."
            out += [(p + "norm1", t + "norm1", (D,), 1.0, 0.02), (p + "norm1.b", t + "norm1.b", (D,), 0.0, 0.02)]
            if isinstance(m, ParallelMixerSpec):
                out += [(p + "mix.left.q.norm", t + "mix.left.q.norm", (m.left.q_rows,), 1.0, 0.02), (p + "mix.left.k.norm", t + "mix.left.k.norm", (m.left.k_rows,), 1.0, 0.02),
                        (p + "mix.right.norm", t + "mix.right.norm", (m.right.out_rows,), 1.0, 0.02), (p + "mix.out", (t + "mix.left.out", t + "mix.right.out"), (D,), 1.0, 0.02)]
            else:
                out += [(p + "mix.norm", t + "mix.norm", (m.out_rows,), 1.0, 0.02), (p + "mix.bias", (t + "mix.i.b", t + "mix.f.b"), (m.heads,), 1.0, 0.5)]
        return out
    out = [("param.embed_tokens", "embed", (spec.vocab, D), 0.0, 1.0), ("param.final_norm", "final.norm", (D,), 1.0, 0.02)]
    for i, l in enumerate(spec.layers):
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.mlp is not None else ()):
            out.append((f"layer_param.{i}.{n}", f"l{i}.{n}", (D,), 1.0, 0.02))
        for n in ("q.norm", "k.norm"):
            out.append((f"layer_param.{i}.mix.{n}", f"l{i}.mix.{n}", (l.mixer.dim,), 1.0, 0.02))
    return out


def tensor_shapes(spec: LayeredSpec) -> dict:
    """name -> shape of every tensor of a model directory."""
    out = {}
    for _, parts, k in weight_plan(spec):
        for name, n in parts:
            if isinstance(name, tuple):
                out.update({t: (n // len(name), k) for t in name})
            elif name is not None:
                out[name] = (n, k)
    for _, name, shape, _, _ in vector_plan(spec):
        out.update({t: shape for t in (name if isinstance(name, tuple) else (name,))})
    for i, l in enumerate(spec.layers):
        if isinstance(l.mixer, AttentionSpec) and l.mixer.diff is not None:
            out.update({f"l{i}.mix.{n}": (l.mixer.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
    return out


def rotation_table(rotary, capacity: int) -> np.ndarray:
    """cos and sin of every position's pairs, [capacity, dims / 2, 2] fp32 (angles in fp64)."""
    a = np.arange(capacity, dtype=np.float64)[:, None] * np.asarray(rotary.frequencies(), np.float64)[None]
    return np.stack([np.cos(a), np.sin(a)], -1).astype(np.float32)


def combination_constant(lq1, lk1, lq2, lk2, diff: float) -> float:
    """lambda of differential attention, one number per layer: exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    a, b = (float(np.dot(np.asarray(x, np.float64), np.asarray(y, np.float64))) for x, y in ((lq1, lk1), (lq2, lk2)))
    return math.exp(a) - math.exp(b) + diff


def _bf16_values(bits) -> np.ndarray:
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


class Sequence:
    """A sequence being decoded: the cache slot it owns and how many positions are in it."""

    def __init__(self, engine: "LayeredEngine", slot: int):
        self.engine, self.slot, self.length = engine, slot, 0

    def append(self, tokens, want=()) -> np.ndarray:
        """Run the sequence's next tokens; logits [len(want), vocab] after the tokens at places ``want``."""
        self.engine.select(self.slot)
        out = self.engine.step(tokens, self.length, want)
        self.length += len(tokens)
        return out

    def close(self):
        if self.slot >= 0:
            self.engine.release(self.slot)
            self.slot = -1


class LayeredEngine(EngineBase):
    def __init__(self, spec: LayeredSpec, capacity: int, device: int = 0, dtype: str = "bfloat16", max_rows: int = MAX_ROWS,
                 runtime: Runtime | None = None, want_logits: bool = True):          # fp32 logits are always kept
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        if capacity < 1 or max_rows < 1:
            raise ValueError("capacity and max_rows must be positive")
        self.spec, self.capacity, self.dtype = spec, capacity, dtype
        self.f32 = int(dtype == "float32")
        self.size = 4 if self.f32 else 2
        self.rt = runtime or Runtime(device)
        self.sm = self.rt.info()["sm"]
        self.max_rows = min(max_rows, capacity)
        self.W: dict[str, int] = {}
        self.V: dict[str, int] = {}
        self.lambdas: dict[int, float] = {}
        self.graph, self.slot = 0, -1
        self.caches: list[list] = []          # per slot: the buffers of every run by role
        self.at: list[int] = []               # per slot: the position that follows what is in it
        self.free: list[int] = []
        self.graphs: dict[int, tuple] = {}    # slot -> (graph, task list)
        self.rows_tasks: dict[tuple, object] = {}
        self._alloc_buffers()
        self.select(self._new_slot())
        self.free.append(self.slot)

    # ------------------------------------------------------------------ buffers
    def _alloc_buffers(self):
        s, rt, D, M, sz, up = self.spec, self.rt, self.spec.hidden, self.max_rows, self.size, TG.round_up
        if s.block == "parallel":
            self._alloc_parallel_buffers()
            return
        mix = [l.mixer for l in s.layers]
        ffs = [l.mlp for l in s.layers if l.mlp is not None]
        runs = len(s.runs())
        self.X = rt.alloc((runs + 1) * D * 4)                 # decode: residual entering each run (+ final)
        self.HB = rt.alloc(max(runs, 1) * D * 4)              # decode: residual after the mixer
        top = max([f.top for f in ffs], default=1)
        tiles = [-(-(m.heads // m.kv_heads * m.maps) // 8) for m in mix]
        part = max(m.kv_heads * t * TG.key_splits(m, self.capacity, self.sm) * 8 * (up(m.vdim, 8) + 2) for m, t in zip(mix, tiles))
        self.scratch = {
            "layer_scratch.qkvg": rt.alloc(max(m.rows for m in mix) * 4), "layer_scratch.attention": rt.alloc(max(m.heads * m.vdim for m in mix) * 4),
            "layer_scratch.mixer_out": rt.alloc(D * 4), "layer_scratch.ff_in": rt.alloc(D * 4), "layer_scratch.ff_out": rt.alloc(D * 4),
            "layer_scratch.router_shared": rt.alloc(max([f.experts + f.shared_ff for f in ffs], default=1) * 4),
            "layer_scratch.expert_act": rt.alloc(max([f.top * f.ff for f in ffs], default=1) * 4), "layer_scratch.chosen": rt.alloc(top * 4),
            "layer_scratch.chosen_weight": rt.alloc(top * 4), "global_scratch.attention_partials": rt.alloc(part * 4),
            "global_scratch.attention_counters": rt.alloc(max(m.kv_heads * t for m, t in zip(mix, tiles)) * 4),
            "global_scratch.logits": rt.alloc(s.vocab * 4), "global_scratch.argmax_scratch": rt.alloc(8 * 1024), "global_scratch.head_counter": rt.alloc(4),
        }
        self.logits = self.scratch["global_scratch.logits"]
        ld, slots = up(D, 64), M * top
        r = {
            "tokens": M * 4, "index": M * 4, "embedding": M * D * 4, "x": M * D * 4, "h": M * ld * sz, "h_wanted": M * ld * sz, "y": M * ld * sz,
            "qkvg": M * max(up(m.rows, 64) for m in mix) * sz, "q": M * max(m.heads * m.maps * up(m.dim, 8) for m in mix) * sz,
            "attention": M * max(up(m.heads * m.vdim, 64) for m in mix) * sz,
            "router": M * max([up(f.experts, 64) for f in ffs], default=1) * 4, "chosen": slots * 4, "chosen_weight": slots * 4, "rank": slots * 4,
            "slot": slots * 4, "count": max([f.experts for f in ffs], default=1) * 4, "offsets": (max([f.experts for f in ffs], default=1) + 1) * 4,
            "h_grouped": slots * ld * sz, "act_grouped": slots * max([up(f.ff, 64) for f in ffs], default=64) * sz, "y_grouped": slots * ld * sz,
            "shared_act": M * max([up(max(f.shared_ff, 1), 64) for f in ffs], default=64) * sz,
        }
        self.scratch.update({"rows_scratch." + k: rt.alloc(n) for k, n in r.items()})
        self.wanted_rows = 0

    def _alloc_parallel_buffers(self):
        s, rt, D, M, sz, up = self.spec, self.rt, self.spec.hidden, self.max_rows, self.size, TG.round_up
        lays, recs = [block_layout(l) for l in s.layers], [TG._recurrence(l)[0] for l in s.layers]
        att = [l.mixer.left for l in s.layers if isinstance(l.mixer, ParallelMixerSpec)]
        ff, ld = max([l.mlp.ff for l in s.layers if l.mlp is not None], default=1), up(D, 64)
        self.X = rt.alloc((len(s.runs()) + 1) * D * 4)
        tiles = [-(-(a.heads // a.kv_heads) // 8) for a in att]
        part = max([a.kv_heads * t * TG.key_splits(a, self.capacity, self.sm) * 8 * (up(a.vdim, 8) + 2) for a, t in zip(att, tiles)], default=1)
        n = {
            "layer_scratch.block": max(l.out_rows for l in lays) * 4, "layer_scratch.attention": max([a.out_rows for a in att], default=1) * 4,
            "layer_scratch.memory": max(r.out_rows for r in recs) * 4, "layer_scratch.sums": 3 * D * 4, "global_scratch.attention_partials": part * 4,
            "global_scratch.attention_counters": max([a.kv_heads * t for a, t in zip(att, tiles)], default=1) * 4, "global_scratch.logits": s.vocab * 4,
            "global_scratch.argmax_scratch": 8 * 1024, "global_scratch.head_counter": 4,
            "rows_scratch.tokens": M * 4, "rows_scratch.index": M * 4, "rows_scratch.embedding": M * D * 4, "rows_scratch.x": M * D * 4, "rows_scratch.h": M * ld * sz,
            "rows_scratch.h_wanted": M * ld * sz, "rows_scratch.y": M * ld * sz, "rows_scratch.y1": M * ld * sz, "rows_scratch.y2": M * ld * sz,
            "rows_scratch.block": M * max(up(l.plain, 64) for l in lays) * sz, "rows_scratch.gate_logits": M * max(max(l.exact - l.plain for l in lays), 1) * 4,
            "rows_scratch.ff": M * up(ff, 64) * sz, "rows_scratch.q": M * max([a.heads * up(a.dim, 8) for a in att], default=1) * sz,
            "rows_scratch.attention": M * max([up(a.out_rows, 64) for a in att], default=1) * sz, "rows_scratch.memory": M * max(up(r.out_rows, 8) for r in recs) * sz,
            "rows_scratch.gated": M * max(up(r.out_rows, 64) for r in recs) * sz, "rows_scratch.runs": max(max(TG.recurrence_scratch(r, M) for r in recs), 1) * 4,
        }
        self.scratch = {k: rt.alloc(v) for k, v in n.items()}
        self.logits, self.wanted_rows = self.scratch["global_scratch.logits"], 0
        tables = {}
        for i, l in enumerate(s.layers):
            rot = l.mixer.left.rotary if isinstance(l.mixer, ParallelMixerSpec) else None
            if rot is not None:
                if rot not in tables:
                    tables[rot] = rt.to_device(rotation_table(rot, self.capacity)) if rot.dims else 0
                self.scratch[f"rotation.{i}"] = tables[rot]
            if isinstance(l.mixer, ParallelMixerSpec):
                d = np.array(l.mixer.right.decay, np.float64)
                with np.errstate(divide="ignore"):
                    self.V[f"layer_param.{i}.mix.right.decay"] = rt.to_device(np.concatenate([np.maximum(np.log(d), -1e4), d]).astype(np.float32))

    def _grow_logits(self, wanted: int):
        if wanted > self.wanted_rows:
            n = min(self.max_rows, max(wanted, 2 * self.wanted_rows))
            if self.wanted_rows:
                N.check(self.rt.L.fk_free(self.rt.h, self.scratch["rows_scratch.logits"]), "fk_free")
            self.scratch["rows_scratch.logits"] = self.rt.alloc(n * self.spec.vocab * 4)
            self.wanted_rows = n
            self.rows_tasks.clear()

    # ------------------------------------------------------------------ cache slots
    def _new_slot(self) -> int:
        up, kv = TG.round_up, []
        for i, _ in self.spec.runs():
            m, bufs = self.spec.layers[i].mixer, {}
            a = m.left if isinstance(m, ParallelMixerSpec) else m if isinstance(m, AttentionSpec) else None
            if a is not None:
                bufs["layer_cache_k"] = self.rt.alloc(a.kv_heads * a.maps * self.capacity * up(a.dim, 8) * self.size)
                bufs["layer_cache_v"] = self.rt.alloc(a.kv_heads * self.capacity * up(a.vdim, 8) * self.size)
            if m is not a:
                bufs["layer_state"] = self.rt.alloc(TG.recurrence_state(TG._recurrence(self.spec.layers[i])[0]) * 4)
            kv.append(bufs)
        self.caches.append(kv)
        self.at.append(0)
        return len(self.caches) - 1

    def select(self, slot: int):
        """Make ``slot`` the one the next steps read and write."""
        if slot != self.slot:
            self.slot = slot
            self.graph, self.replay = self.graphs.get(slot, (0, []))
            self.tasks = self.replay

    def open_sequence(self) -> Sequence:
        return Sequence(self, self.free.pop() if self.free else self._new_slot())

    def release(self, slot: int):
        if slot in self.free or not 0 <= slot < len(self.caches):
            raise ValueError(f"cache slot {slot} is not in use")
        self.free.append(slot)

    # ------------------------------------------------------------------ tensors
    def load_from(self, provider):
        """``provider(name, shape)`` -> bf16 bit patterns of a tensor."""
        rt = self.rt
        for role, parts, k in weight_plan(self.spec):
            kp = TG.round_up(k, 64)
            wid, row = rt.weight_alloc(sum(n for _, n in parts), kp, 16), 0
            for tensor, n in parts:
                if tensor is None:
                    a = np.zeros((n, k), np.uint16)
                elif isinstance(tensor, tuple):
                    a = np.stack([np.asarray(provider(x, (n // len(tensor), k)), np.uint16) for x in tensor], 1).reshape(n, k)
                else:
                    a = np.asarray(provider(tensor, (n, k)), np.uint16)
                if kp != k:
                    a = np.concatenate([a, np.zeros((n, kp - k), np.uint16)], 1)
                rt.weight_upload_rows(wid, row, a)
                row += n
            rt.weight_keep_rows(wid)
            self.W[role] = wid
        for role, tensor, shape, _, _ in vector_plan(self.spec):
            a = [np.asarray(provider(x, shape), np.uint16).reshape(-1) for x in (tensor if isinstance(tensor, tuple) else (tensor,))]
            self.V[role] = rt.to_device(np.concatenate(a))
        for i, l in enumerate(self.spec.layers):
            m, v = l.mixer, []
            if not isinstance(m, AttentionSpec):
                continue
            if m.diff is not None:
                v = [_bf16_values(provider(f"l{i}.mix.{n}", (m.dim,))) for n in ("lq1", "lk1", "lq2", "lk2")]
            self.lambdas[i] = combination_constant(*v, m.diff) if v else 0.0
        rt.sync()

    def load_synthetic(self):
        """Every tensor generated on the device from its named stream (columns must be whole multiples of 64)."""
        s, rt = self.spec, self.rt
        for role, parts, k in weight_plan(s):
            if k % 64:
                raise ValueError(f"synthetic weights need input sizes in multiples of 64 ({role}: {k})")
            wid, row = rt.weight_alloc(sum(n for _, n in parts), k, 16), 0
            for tensor, n in parts:
                if tensor is None:
                    rt.weight_upload_rows(wid, row, np.zeros((n, k), np.uint16))
                else:                       # tensors taken in turn are one stream of rows here
                    rt.weight_synth_rows(wid, row, n, stream_id(s.seed, tensor if isinstance(tensor, str) else "+".join(tensor)), 1.0 / math.sqrt(k), k, 0, 0)
                row += n
            rt.weight_keep_rows(wid)
            self.W[role] = wid
        for role, tensor, shape, mean, std in vector_plan(s):
            n, names = int(np.prod(shape)), tensor if isinstance(tensor, tuple) else (tensor,)
            self.V[role] = rt.alloc(n * len(names) * 2)
            for j, name in enumerate(names):
                rt.synth_normal(self.V[role] + j * n * 2, stream_id(s.seed, name), 0, n, mean, std)
        self.lambdas = {i: l.mixer.diff or 0.0 for i, l in enumerate(s.layers) if isinstance(l.mixer, AttentionSpec)}
        rt.sync()

    def prefill_kv_synthetic(self, ctx: int):
        """Positions [0, ctx) of the selected slot's bf16 caches from N(0, 1) streams; states are left as they are."""
        mixers = [l.mixer.left if isinstance(l.mixer, ParallelMixerSpec) else l.mixer for l in self.spec.layers]
        if self.f32 or any(m.dim % 8 or m.vdim % 8 for m in mixers if isinstance(m, AttentionSpec)):
            raise ValueError("synthetic cache rows are bf16 with head sizes in multiples of 8")
        self.at[self.slot] = ctx
        for run, (i, _) in enumerate(self.spec.runs()):
            m, bufs = mixers[i], self.caches[self.slot][run]
            if not isinstance(m, AttentionSpec):
                continue
            for which, heads, d, p in (("k", m.kv_heads * m.maps, m.dim, bufs["layer_cache_k"]), ("v", m.kv_heads, m.vdim, bufs["layer_cache_v"])):
                for hh in range(heads):
                    self.rt.synth_normal(p + hh * self.capacity * d * 2, stream_id(self.spec.seed, f"runs.{run}.cache_{which}"), hh * 1048576 * d, ctx * d, 0.0, 1.0)
        self.rt.sync()

    # ------------------------------------------------------------------ task graph
    def task_graph(self) -> dict:
        return TG.emit_layered(self.spec, self.capacity, self.lambdas, self.f32, self.sm)

    def _resolve(self, role: str) -> int:
        p = role.split(".")
        if role in self.W:
            return self.W[role]
        if role in self.V:
            return self.V[role]
        if role in self.scratch:
            return self.scratch[role]
        if p[0] in ("layer_cache_k", "layer_cache_v", "layer_state"):
            return self.caches[self.slot][int(p[1])][p[0]]
        if p[1:2] == ["block"]:                                   # a part of the joint projection: <layer>.<part>
            l = self.spec.layers[int(p[2])]
            lay, rec, size = block_layout(l), TG._recurrence(l)[0], 4 if p[0] == "layer_scratch" else self.size
            first = {"q": lay.parts["recurrence"], "k": lay.parts["recurrence"] + rec.heads * rec.dim, "v": lay.parts["recurrence"] + 2 * rec.heads * rec.dim, **lay.parts}
            return self.scratch[p[0] + ".block"] + first[p[3]] * size
        if role.startswith("global_scratch.x_in."):
            return self.X + int(p[2]) * self.spec.hidden * 4
        if p[0] == "layer_scratch" and p[-1] == "h_attn":
            return self.HB + int(p[1]) * self.spec.hidden * 4
        if role.startswith("layer_scratch.shared_act."):          # rows after the router's in the joint product
            return self.scratch["layer_scratch.router_shared"] + self.spec.layers[int(p[2])].mlp.experts * 4
        if role.startswith("rows_scratch.gate."):                 # columns after q | k | v
            m = self.spec.layers[int(p[2])].mixer
            return self.scratch["rows_scratch.qkvg"] + (m.rows - m.heads) * self.size
        raise KeyError(f"unknown task-graph role {role!r}")

    def capture(self) -> int:
        super().capture()
        self.graphs[self.slot] = (self.graph, self.replay)
        return self.graph

    def rows_dispatches(self, rows: int, wanted: int, greedy: bool) -> list:
        tasks = TG.layered_rows_tasks(self.spec, self.capacity, self.lambdas, rows, wanted, greedy, self.f32)
        return [N.Task.make(t["kind"], t["layer"], {s: self._resolve(r) for s, r in t["bufs"].items()}, t["iargs"], t["fargs"]) for t in tasks]

    # ------------------------------------------------------------------ steps
    def _check(self, tokens, base_offset: int):
        toks = np.ascontiguousarray(tokens, np.uint32)
        if toks.ndim != 1 or not len(toks):
            raise ValueError("a step needs at least one token")
        if int(toks.max()) >= self.spec.vocab:
            raise ValueError(f"token id {int(toks.max())} is outside the vocabulary ({self.spec.vocab})")
        self._check_place(base_offset, len(toks))
        return toks

    def _check_place(self, base_offset: int, count: int):
        if base_offset < 0 or base_offset + count > self.capacity:
            raise ValueError(f"positions {base_offset} .. {base_offset + count - 1} do not fit the cache ({self.capacity})")
        if self.spec.recurrent and base_offset not in (0, self.at[self.slot]):
            raise ValueError(f"the state of this sequence stands at position {self.at[self.slot]}: it can be continued there or started again, not at {base_offset}")

    def _run_rows(self, toks, base_offset: int, want, greedy: bool):
        rt, key = self.rt, (self.slot, len(toks), len(want), greedy)
        self._grow_logits(len(want))
        if key not in self.rows_tasks:
            if len(self.rows_tasks) > 64:
                self.rows_tasks.clear()
            tasks = self.rows_dispatches(len(toks), len(want), greedy)
            self.rows_tasks[key] = (N.Task * len(tasks))(*tasks)
        arr = self.rows_tasks[key]
        self.at[self.slot] = base_offset + len(toks)
        rt.upload(self.scratch["rows_scratch.tokens"], toks)
        if len(want):
            rt.upload(self.scratch["rows_scratch.index"], np.asarray(want, np.uint32))
        rt.state_set(0, base_offset)          # the tokens come from their buffer
        N.check(rt.L.fk_launch_batch(rt.h, arr, len(arr)), "fk_launch_batch")
        token, _, err = rt.state_get()
        if err:
            raise N.FusekitError(f"device error word {err:#x}")
        return token

    def step(self, tokens, base_offset: int, want=()) -> np.ndarray:
        """Run ``tokens`` at positions base_offset .. of the selected slot; logits (fp32) after the tokens at places ``want``."""
        toks, want = self._check(tokens, base_offset), [int(w) for w in want]
        if want and not (0 <= min(want) and max(want) < len(toks)):
            raise ValueError("wanted places lie outside the step's tokens")
        out = np.empty((len(want), self.spec.vocab), np.float32)
        for c0 in range(0, len(toks), self.max_rows):
            part = toks[c0:c0 + self.max_rows]
            here = [j for j, w in enumerate(want) if c0 <= w < c0 + len(part)]
            if len(part) == 1:
                self.decode_chunk(base_offset + c0, int(part[0]), 1)
                if here:
                    out[here] = self.last_logits()
                continue
            self._run_rows(part, base_offset + c0, [want[j] - c0 for j in here], False)
            if here:
                out[here] = self.rt.download(self.scratch["rows_scratch.logits"], (len(here), self.spec.vocab), np.float32)
        return out

    def prefill(self, tokens, base_offset: int = 0) -> int:
        """Run a prompt through the selected slot; the greedy token after its last position."""
        toks, nxt = self._check(tokens, base_offset), 0
        for c0 in range(0, len(toks), self.max_rows):
            part = toks[c0:c0 + self.max_rows]
            last = c0 + len(part) == len(toks)
            if len(part) == 1:
                nxt = int(self.decode_chunk(base_offset + c0, int(part[0]), 1)[0][0])
            else:
                nxt = self._run_rows(part, base_offset + c0, [len(part) - 1] if last else [], last)
        return int(nxt)

    def decode_chunk(self, base_offset: int, seed_token: int, count: int):
        self._check_place(base_offset, count)
        self.at[self.slot] = base_offset + count
        return super().decode_chunk(base_offset, seed_token, count)

    def last_logits(self) -> np.ndarray:
        """fp32 logits of the last decoded position."""
        return self.rt.download(self.logits, (self.spec.vocab,), np.float32)

    def residual_stream(self) -> np.ndarray:
        """fp32 residual entering every run of the last decoded position, and the final one, [runs + 1, D] (a repeated pass enters
        with the embedding output added)."""
        return self.rt.download(self.X, (len(self.spec.runs()) + 1, self.spec.hidden), np.float32)

    def complete(self, prompt, max_tokens: int, *args, **kw) -> np.ndarray:
        """A completion in a slot of its own (see EngineBase.complete)."""
        seq = self.open_sequence()
        try:
            self.select(seq.slot)
            return super().complete(prompt, max_tokens, *args, **kw)
        finally:
            seq.close()
