"""The compiler -> runtime contract of the decode path: a ``task_graph.json`` in the reference's v2 shape.

The reference writes this file from its fused task graph (src/codegen/task_graph_json.rs:33-226) and its runtime
reads it back (src/runtime/plan.rs:39-164, python/fusekit_runtime/dispatch.py:318-329).  Capture needs MLX, so here
the graph is produced from the model shape: one task per fused decode kernel, buffers named by the reference's
role strings (``slot_role_key``, src/codegen/kernels/mod.rs:5531-5576), in replay order (embed -> per layer
RmsNormQkv, SDPA, LinearResidual, gate/up chain, LinearResidual -> final head; task_graph_json.rs:1619-1664).
``DecodeEngine.build_dispatches`` resolves exactly this structure to device addresses, so the JSON is the list the
GPU replays, not a description on the side.
"""
from __future__ import annotations

import math

from .model_spec import ModelSpec, ParallelMixerSpec, block_layout, round_up

VERSION = 2
KINDS = ["step_init", "embed_lookup_decode", "rmsnorm_qkv", "qk_norm_rope_store", "sdpa_decode", "linear_residual",
         "rmsnorm_gateup_act", "final_rmsnorm_lm_head", "argmax_finalize", "allreduce", "residual_add", "rmsnorm_rows",
         "rope_store_rows", "argmax_rows", "kv_store_quant", "sdpa_decode_quant", "embed_rows", "residual_norm_rows", "linear_rows",
         "qk_norm_store_rows", "attention_rows", "moe_route_rows", "norm_linear", "attention_decode", "moe_up", "moe_down", "argmax_row",
         "block_norm_rows", "block_linear_rows", "rotary_store_rows", "window_attention_rows", "window_attention_decode", "recurrence_rows",
         "recurrence_decode", "norm_gate_rows", "segment_linear"]
KERNEL = {k: "fusekit_" + k for k in KINDS}
(K_STEP, K_EMBED, K_QKV, K_QKNORM, K_SDPA, K_LIN, K_GATEUP, K_HEAD, K_ARGMAX, K_ALLREDUCE, K_RESADD, K_NORMROWS, K_ROPEROWS,
 K_ARGMAXROWS, K_KVQ, K_SDPAQ, K_EMBEDROWS, K_RESNORM, K_LINROWS, K_QKSTORE, K_ATTROWS, K_ROUTE, K_NORMLIN, K_ATTDEC, K_MOEUP,
 K_MOEDOWN, K_ARGMAXROW, K_BLOCKNORM, K_BLOCKLIN, K_ROTSTORE, K_WINROWS, K_WINDEC, K_RECROWS, K_RECDEC, K_NORMGATE, K_SEGLIN) = range(36)


def _bf16_round(v: float) -> float:
    import struct
    u = struct.unpack("<I", struct.pack("<f", v))[0]
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return struct.unpack("<f", struct.pack("<I", u))[0]


def emit(spec: ModelSpec, capacity: int, tp_rank: int = 0, tp_size: int = 1, fused_weights: bool = True,
         want_logits: bool = False, embed_bits: int = 16, tp_exchange: str = "allreduce", kv_bits: int = 0,
         fuse_attention: bool = False, act_digits: bool = False) -> dict:
    """Build the v2 task graph of one decode step for `spec` (one tensor-parallel rank of it).

    `fused_weights`: weights in the streaming layout (gate/up paired, residual add after an all-reduce fused into the next
    norm-first kernel); False describes the generic kernels on MLX-layout rows.
    `tp_exchange`: how the partial rows of the row-split projections meet -- "allreduce": an all-reduce task after each
    (library collective or the stand-alone peer kernel); "peer": no task of its own, the projection pushes its partial rows
    into every rank's arena and the next norm-first kernel sums them (exchange site 2l for o_proj, 2l + 1 for down_proj of
    layer l, 2L for the argmax keys of the vocabulary-sharded head).
    `kv_bits`: 4 or 8 = quantised KV cache (Qwen-shaped layers, one GPU): the QKV task writes raw projections, a
    kv_store_quant task rotates and quantises, sdpa_decode_quant attends the packed cache
    (src/codegen/kernels/rope_kv_cache_store_decode_quant.rs, sdpa_decode_quant.rs).
    `fuse_attention`: Qwen-shaped layers with the streaming layout and a bf16 cache: no sdpa_decode task, the QKV task attends
    the cache in its tail (iarg 7, slot 7 = attention output, slot 8 = scratch, farg 2 = scale).
    `act_digits`: one GPU, Qwen-shaped layers, 4/8-bit streaming layout: the gate/up task also leaves its output as the integer
    digits down_proj stages (slot 5 of both tasks, `layer_scratch.silu_up_digits`), so down_proj copies instead of converting."""
    s, hd, H = spec, spec.head_dim, spec.hidden
    nq, nkv, inter, vocab = s.n_q // tp_size, s.n_kv // tp_size, s.inter // tp_size, s.vocab // tp_size
    tp = tp_size > 1
    fused = fused_weights
    peer = tp and tp_exchange == "peer"
    if kv_bits and (kv_bits not in (4, 8) or s.arch != "qwen2" or tp):
        raise ValueError("the quantised KV cache is wired for Qwen-shaped layers on one GPU, 4 or 8 bits")
    attend = bool(fuse_attention) and s.arch == "qwen2" and fused and not kv_bits and not tp and hd in (64, 128) and s.n_q // s.n_kv <= 8
    if peer and not fused:
        raise ValueError("the fused peer exchange needs the streaming weight layout")
    if peer and 2 * s.n_layers + 1 > 160:
        raise ValueError("the fused peer exchange has 160 sites: at most 79 layers")
    tasks: list[dict] = []

    def add(kind, layer, bufs, iargs, fargs=()):
        tasks.append({"kind": kind, "layer": layer, "bufs": {int(k): v for k, v in bufs.items() if v}, "iargs": [int(v) for v in iargs],
                      "fargs": [float(v) for v in fargs]})

    x = lambda l: f"global_scratch.x_in.{l}"           # residual stream entering layer l (l = n_layers: final)
    hb = lambda l: f"layer_scratch.{l}.h_attn"
    lp = lambda l, rel: f"layer_param.{l}.{rel}"
    gateup = (lambda l: {2: lp(l, "mlp.gate_up_proj")}) if fused else (lambda l: {2: lp(l, "mlp.gate_proj"), 3: lp(l, "mlp.up_proj")})
    emb_scale = _bf16_round(math.sqrt(H)) if s.arch == "gemma3" else 1.0      # embed_lookup_decode.rs OUTPUT_SCALE
    if embed_bits in (4, 8):      # quantised embedding rows, dequantised in the gather (embed_lookup_decode.rs:40-61 signature)
        add(K_EMBED, -1, {0: "param.embed_tokens", 1: x(0), 2: "param.embed_tokens.scales", 3: "param.embed_tokens.biases"},
            [H, 1, s.vocab, embed_bits], [emb_scale])
    else:
        add(K_EMBED, -1, {0: "param.embed_tokens", 1: x(0)}, [H, 1, s.vocab], [emb_scale])
    scale = 1.0 / math.sqrt(hd)
    for l in range(s.n_layers):
        cap, theta = s.layer_capacity(l, capacity), s.layer_theta(l)
        ck, cv = f"layer_cache_k.{l}", f"layer_cache_v.{l}"
        if s.arch == "qwen2":
            x_in, pend, pull = x(l), {}, 0
            if tp and l > 0 and fused and peer:            # x[l] = T(sum of the ranks' down_proj partials + h[l-1])
                x_in, pend, pull = hb(l - 1), {11: x(l)}, 2 * (l - 1) + 2
            elif tp and l > 0 and fused:                   # x[l] = T(all-reduced down_proj + h[l-1])
                x_in, pend = hb(l - 1), {9: "global_scratch.tp_partial_b", 11: x(l)}
            if kv_bits:
                cq = {n: f"layer_cache_{n}.{l}" for n in ("k", "v", "k_scales", "k_biases", "v_scales", "v_biases")}
                add(K_QKV, l, {0: x_in, 1: lp(l, "input_layernorm.weight"), 2: lp(l, "self_attn.qkv_proj"), 3: lp(l, "self_attn.qkv_proj.bias"),
                               4: "layer_scratch.q_buf", 7: "layer_scratch.k_buf", 8: "layer_scratch.v_buf"}, [H, nq, nkv, hd, cap, 0], [s.eps, theta])
                add(K_KVQ, l, {0: "layer_scratch.q_buf", 1: "layer_scratch.k_buf", 2: "layer_scratch.v_buf", 3: cq["k"], 4: cq["v"], 5: cq["k_scales"],
                               6: cq["k_biases"], 7: cq["v_scales"], 8: cq["v_biases"]}, [nq, nkv, hd, cap, kv_bits], [0.0, theta])
            elif attend:
                add(K_QKV, l, {0: x_in, 1: lp(l, "input_layernorm.weight"), 2: lp(l, "self_attn.qkv_proj"), 3: lp(l, "self_attn.qkv_proj.bias"),
                               4: "layer_scratch.q_buf", 5: ck, 6: cv, 7: "layer_scratch.sdpa_buf", 8: "global_scratch.attend_scratch", **pend},
                    [H, nq, nkv, hd, cap, 1, pull, 1], [s.eps, theta, 1.0 / math.sqrt(hd)])
            else:
                add(K_QKV, l, {0: x_in, 1: lp(l, "input_layernorm.weight"), 2: lp(l, "self_attn.qkv_proj"), 3: lp(l, "self_attn.qkv_proj.bias"),
                               4: "layer_scratch.q_buf", 5: ck, 6: cv, **pend}, [H, nq, nkv, hd, cap, 1, pull], [s.eps, theta])
        else:
            x_in, pend = x(l), {}
            if l > 0:                                      # Gemma: x[l] = T(h[l-1] + rmsnorm(down_out[l-1]))
                x_in, pend = hb(l - 1), {9: f"layer_scratch.{l-1}.out_buf", 10: lp(l - 1, "post_feedforward_layernorm.weight"), 11: x(l)}
            add(K_QKV, l, {0: x_in, 1: lp(l, "input_layernorm.weight"), 2: lp(l, "self_attn.qkv_proj"), 4: "layer_scratch.q_buf",
                           7: "layer_scratch.k_buf", 8: "layer_scratch.v_buf", **pend}, [H, nq, nkv, hd, cap, 0], [s.eps, theta])
            add(K_QKNORM, l, {0: "layer_scratch.q_buf", 1: "layer_scratch.k_buf", 2: "layer_scratch.v_buf", 3: lp(l, "self_attn.q_norm.weight"),
                              4: lp(l, "self_attn.k_norm.weight"), 5: ck, 6: cv}, [nq, nkv, hd, cap], [s.eps, theta])
        if kv_bits:
            add(K_SDPAQ, l, {0: "layer_scratch.q_buf", 1: cq["k"], 2: cq["v"], 3: "layer_scratch.sdpa_buf", 4: "global_scratch.sdpa_partials",
                             5: "global_scratch.sdpa_counter", 6: cq["k_scales"], 7: cq["k_biases"], 8: cq["v_scales"], 9: cq["v_biases"]},
                [nq, nkv, hd, cap, kv_bits], [scale])
        elif not attend:
            add(K_SDPA, l, {0: "layer_scratch.q_buf", 1: ck, 2: cv, 3: "layer_scratch.sdpa_buf", 4: "global_scratch.sdpa_partials",
                            5: "global_scratch.sdpa_counter"}, [nq, nkv, hd, cap], [scale])
        ko = nq * hd
        if s.arch == "qwen2" and not tp:
            add(K_LIN, l, {0: "layer_scratch.sdpa_buf", 1: lp(l, "self_attn.o_proj"), 2: x(l), 3: hb(l)}, [ko, H])
            dig = {5: "layer_scratch.silu_up_digits"} if (act_digits and fused and s.bits in (4, 8) and inter % 64 == 0) else {}
            add(K_GATEUP, l, {0: hb(l), 1: lp(l, "post_attention_layernorm.weight"), **gateup(l), 4: "layer_scratch.silu_up", **dig}, [H, inter, s.act], [s.eps])
            add(K_LIN, l, {0: "layer_scratch.silu_up", 1: lp(l, "mlp.down_proj"), 2: hb(l), 3: x(l + 1), **dig}, [inter, H])
        elif s.arch == "qwen2" and peer:
            # row-split o/down with the exchange fused in: the projection pushes fp32 partial rows to every rank (site in i3),
            # the next norm-first kernel waits for all ranks, sums in rank order and adds the residual (site in its last iarg)
            add(K_LIN, l, {0: "layer_scratch.sdpa_buf", 1: lp(l, "self_attn.o_proj")}, [ko, H, 0, 2 * l + 1])
            add(K_GATEUP, l, {0: x(l), 11: hb(l), 1: lp(l, "post_attention_layernorm.weight"), **gateup(l), 4: "layer_scratch.silu_up"},
                [H, inter, s.act, 0, 2 * l + 1], [s.eps])
            add(K_LIN, l, {0: "layer_scratch.silu_up", 1: lp(l, "mlp.down_proj")}, [inter, H, 0, 2 * l + 2])
        elif s.arch == "qwen2":
            # row-split o/down: fp32 partial -> all-reduce over the ranks; the residual add rides in the next norm-first
            # kernel's prologue (streamed weights) or in a small kernel (generic weights)
            pa, pb = "global_scratch.tp_partial_a", "global_scratch.tp_partial_b"
            add(K_LIN, l, {0: "layer_scratch.sdpa_buf", 1: lp(l, "self_attn.o_proj"), 4: pa}, [ko, H])
            add(K_ALLREDUCE, l, {0: pa}, [H, 0])
            if not fused:
                add(K_RESADD, l, {0: pa, 1: x(l), 2: hb(l)}, [H])
            gin = {0: x(l), 9: pa, 11: hb(l)} if fused else {0: hb(l)}
            add(K_GATEUP, l, {**gin, 1: lp(l, "post_attention_layernorm.weight"), **gateup(l), 4: "layer_scratch.silu_up"}, [H, inter, s.act], [s.eps])
            add(K_LIN, l, {0: "layer_scratch.silu_up", 1: lp(l, "mlp.down_proj"), 4: pb}, [inter, H])
            add(K_ALLREDUCE, l, {0: pb}, [H, 0])
            if not fused:
                add(K_RESADD, l, {0: pb, 1: hb(l), 2: x(l + 1)}, [H])
        else:
            # Gemma-shaped: o_proj plain; post-attention norm + residual + pre-ffn norm in the gate/up prologue
            add(K_LIN, l, {0: "layer_scratch.sdpa_buf", 1: lp(l, "self_attn.o_proj"), 3: "layer_scratch.o_buf"}, [ko, H])
            add(K_GATEUP, l, {0: x(l), 1: lp(l, "pre_feedforward_layernorm.weight"), **gateup(l), 4: "layer_scratch.silu_up",
                              9: "layer_scratch.o_buf", 10: lp(l, "post_attention_layernorm.weight"), 11: hb(l)}, [H, inter, s.act], [s.eps])
            add(K_LIN, l, {0: "layer_scratch.silu_up", 1: lp(l, "mlp.down_proj"), 3: f"layer_scratch.{l}.out_buf"}, [inter, H])
    L = s.n_layers
    x_fin, pend = x(L), {}
    if s.arch == "gemma3":
        x_fin, pend = hb(L - 1), {9: f"layer_scratch.{L-1}.out_buf", 10: lp(L - 1, "post_feedforward_layernorm.weight"), 11: x(L)}
    elif tp and fused and peer:
        x_fin, pend = hb(L - 1), {11: x(L)}
    elif tp and fused:
        x_fin, pend = hb(L - 1), {9: "global_scratch.tp_partial_b", 11: x(L)}
    add(K_HEAD, -1, {0: x_fin, 1: "param.final_norm", 2: "param.lm_head", 3: "global_scratch.logits" if want_logits else None,
                     4: "global_scratch.argmax_scratch", 5: "global_scratch.head_counter", **pend},
        [H, vocab, tp_rank * vocab, 0 if tp else 1] + ([2 * (L - 1) + 2, 2 * L + 1] if (tp and fused and peer) else []), [s.eps])
    if tp and not (fused and peer):
        add(K_ALLREDUCE, -1, {0: "global_scratch.argmax_scratch"}, [1, 1])
        add(K_ARGMAX, -1, {4: "global_scratch.argmax_scratch"}, [1])

    out_slots = {K_EMBED: [1], K_QKV: [4, 5, 6, 7, 8, 11], K_QKNORM: [0, 5, 6], K_SDPA: [3, 4, 5], K_LIN: [3, 4], K_GATEUP: [4, 5, 11],
                 K_HEAD: [3, 4, 5, 11], K_ARGMAX: [], K_ALLREDUCE: [0], K_RESADD: [2], K_KVQ: [0, 3, 4, 5, 6, 7, 8], K_SDPAQ: [3, 4, 5]}
    return _envelope(tasks, out_slots, {"chip": "b200", "arch": "sm_100a", "tensor_parallel": tp_size, "rank": tp_rank, "bits": s.bits,
                                        "launch": "grid and block sizes are chosen by the runtime from the SM count (plan_shape)"})


def _envelope(tasks: list, out_slots: dict, target: dict) -> dict:
    """The v2 document around a task list: tasks with bindings, a linear event chain, layer groups, the decode pipeline."""
    jtasks, groups = [], {}
    for i, t in enumerate(tasks):
        ins, outs, extra = [], [], []
        for slot, role in sorted(t["bufs"].items()):
            if role.startswith(("param.", "layer_param.")):
                ins.append({"role": "external", "tensor_id": len(ins), "source_path": "model." + role.split(".", 1)[1], "role_name": role})
            elif slot in out_slots[t["kind"]]:
                outs.append({"role": "scratch", "scratch_id": slot, "role_name": role})
            else:
                ins.append({"role": "scratch", "scratch_id": slot, "role_name": role})
            extra.append({"slot": slot, "role": role})
        if t["kind"] not in (K_ALLREDUCE, K_RESADD):
            extra += [{"slot": 100, "role": "token_id_in" if t["kind"] in (K_EMBED, K_EMBEDROWS) else "layer_offset"}]
        if t["kind"] in (K_HEAD, K_ARGMAX) or (t["kind"] == K_NORMLIN and 9 in t["bufs"]):
            extra += [{"slot": 101, "role": "next_token_out"}]
        jt = {"id": i, "fusion_id": i, "kernel": KERNEL[KINDS[t["kind"]]], "kind": t["kind"], "grid_threads": [0, 1, 1], "threadgroup": [0, 1, 1],
              "inputs": ins, "outputs": outs, "extra_bindings": extra, "depends_on": [i - 1] if i else [], "trigger_event": i,
              "iargs": t["iargs"], "fargs": t["fargs"]}
        if t["layer"] >= 0:
            jt["layer_idx"] = t["layer"]
        jtasks.append(jt)
        region = "embed" if t["kind"] in (K_EMBED, K_EMBEDROWS) else (f"layer.{t['layer']}" if t["layer"] >= 0 else "post")
        groups.setdefault(region, []).append(i)
    return {
        "version": VERSION, "active_m": 1, "tasks": jtasks,
        "events": [{"id": i, "num_triggers": 1, "fires": [i + 1] if i + 1 < len(jtasks) else []} for i in range(len(jtasks))],
        "scratch_buffers": [], "initial_tasks": [0], "model_params": [],
        "layer_groups": [{"region": r, "task_ids": ids} for r, ids in groups.items()],
        "decode_pipeline": list(range(len(jtasks))),
        "decode_capabilities": {"dispatchable": True, "reasons": []},
        "target": target,
    }


# ------------------------------------------------------------------ layered decoders (model_spec.LayeredSpec)
def _task(tasks, kind, layer, bufs, iargs, fargs=()):
    tasks.append({"kind": kind, "layer": layer, "bufs": {int(k): v for k, v in bufs.items() if v}, "iargs": [int(v) for v in iargs],
                  "fargs": [float(v) for v in fargs]})


def key_splits(mixer, capacity: int, sm: int) -> int:
    """Blocks the keys of a decode step are split over: two blocks per SM over all kv heads, at most 64 (the last
    block to finish folds the others' results) and at least 64 keys of capacity each."""
    tiles = -(-(mixer.heads // mixer.kv_heads * mixer.maps) // 8)
    return max(1, min(-(-2 * sm // (mixer.kv_heads * tiles)), -(-mixer.visible(capacity) // 64), 64))


def layered_decode_tasks(spec, capacity: int, lambdas: dict, dtype: int = 0, sm: int = 148) -> list:
    """One decoded position: per layer run q|k|v|gate projection (previous sublayer's post-norm, residual add and this one's
    pre-norm in its prologue), attention with the q/k norm and the cache store in its prologue, output projection, router and
    shared up-projection in one product, the chosen experts' up- and down-projections; then the head with the greedy choice."""
    if spec.block == "parallel":
        return parallel_decode_tasks(spec, capacity, dtype, sm)
    D, eps, t = spec.hidden, spec.eps, []
    x = lambda r: f"global_scratch.x_in.{r}"
    _task(t, K_EMBEDROWS, -1, {0: "param.embed_tokens", 1: x(0)}, [D, 1, spec.vocab])
    cur, pend, post = x(0), None, None
    for run, (i, again) in enumerate(spec.runs()):
        m, f, lp = spec.layers[i].mixer, spec.layers[i].mlp, f"layer_param.{i}."
        xo = x(run) if run else None
        _task(t, K_NORMLIN, run, {0: cur, 1: pend, 2: post, 3: x(0) if again else None, 4: xo, 5: lp + "norm1", 6: lp + "mix.qkvg", 7: "layer_scratch.qkvg"},
              [D, m.rows, 0, 0], [eps])
        cur = xo or cur
        _task(t, K_ATTDEC, run, {0: "layer_scratch.qkvg", 1: lp + "mix.q.norm", 2: lp + "mix.k.norm", 3: f"layer_cache_k.{run}", 4: f"layer_cache_v.{run}",
                                 5: "layer_scratch.attention", 6: "global_scratch.attention_partials", 7: "global_scratch.attention_counters"},
              [m.heads, m.kv_heads, m.dim, m.vdim, capacity, 1, dtype | m.maps << 8, key_splits(m, capacity, sm)], [m.scale, lambdas[i], m.diff or 0.0, eps])
        _task(t, K_NORMLIN, run, {0: "layer_scratch.attention", 6: lp + "mix.o", 7: "layer_scratch.mixer_out"}, [m.heads * m.vdim, D, 0, 0], [eps])
        pend, post = "layer_scratch.mixer_out", lp + "norm1b"
        if f is None:
            continue
        act = 2
        _task(t, K_NORMLIN, run, {0: cur, 1: pend, 2: post, 4: f"layer_scratch.{run}.h_attn", 5: lp + "norm2", 6: lp + "mlp.router_shared",
                                  7: "layer_scratch.router_shared", 8: "layer_scratch.ff_in"}, [D, f.experts + f.shared_ff, act, f.experts], [eps])
        cur = f"layer_scratch.{run}.h_attn"
        _task(t, K_MOEUP, run, {0: "layer_scratch.router_shared", 1: "layer_scratch.ff_in", 2: lp + "mlp.experts_up", 3: "layer_scratch.expert_act",
                                4: "layer_scratch.chosen", 5: "layer_scratch.chosen_weight"}, [D, f.experts, f.top, f.ff, act])
        _task(t, K_MOEDOWN, run, {0: "layer_scratch.expert_act", 1: "layer_scratch.chosen", 2: "layer_scratch.chosen_weight", 3: lp + "mlp.experts_down",
                                  4: f"layer_scratch.shared_act.{i}" if f.shared_ff else None, 5: lp + "mlp.shared_down" if f.shared_ff else None,
                                  6: "layer_scratch.ff_out"}, [D, f.experts, f.top, f.ff, f.shared_ff])
        pend, post = "layer_scratch.ff_out", lp + "norm2b"
    _task(t, K_NORMLIN, -1, {0: cur, 1: pend, 2: post, 4: x(len(spec.runs())), 5: "param.final_norm", 6: "param.lm_head", 7: "global_scratch.logits",
                             9: "global_scratch.argmax_scratch", 10: "global_scratch.head_counter"}, [D, spec.vocab, 0, 0], [eps])
    return t


def layered_rows_tasks(spec, capacity: int, lambdas: dict, rows: int, wanted: int, greedy: bool, dtype: int = 0) -> list:
    """``rows`` consecutive positions: the same layers on row kernels; logits of the ``wanted`` rows of the index buffer, and with
    ``greedy`` the token after the first of them (the position then advances by ``rows``)."""
    if spec.block == "parallel":
        return parallel_rows_tasks(spec, capacity, rows, wanted, greedy, dtype)
    D, V, M, eps, t = spec.hidden, spec.vocab, rows, spec.eps, []
    ld = round_up(D, 64)
    emb, xb, h = "rows_scratch.embedding", "rows_scratch.x", "rows_scratch.h"
    _task(t, K_EMBEDROWS, -1, {0: "param.embed_tokens", 1: emb, 2: "rows_scratch.tokens"}, [D, M, V])
    cur, pend, post, top = emb, {}, None, 0

    def linear(run, x, w, y, n, ldx, ldy, act=0, row0=0, f32=0, m=M, grouped=None, experts=0):
        _task(t, K_LINROWS, run, {0: x, 1: w, 2: y, 3: grouped}, [m, row0, n, ldx, ldy, dtype, act | f32 << 8, experts])

    for run, (i, again) in enumerate(spec.runs()):
        m, f, lp = spec.layers[i].mixer, spec.layers[i].mlp, f"layer_param.{i}."
        _task(t, K_RESNORM, run, {0: cur, 2: post, 3: emb if again else None, 4: xb if run else None, 5: lp + "norm1", 6: h, **pend},
              [D, M, dtype, ld, top, ld], [eps])
        cur = xb if run else cur
        ldq, ldo = round_up(m.rows, 64), round_up(m.heads * m.vdim, 64)
        linear(run, h, lp + "mix.qkvg", "rows_scratch.qkvg", m.rows, ld, ldq)
        _task(t, K_QKSTORE, run, {0: "rows_scratch.qkvg", 1: lp + "mix.q.norm", 2: lp + "mix.k.norm", 3: "rows_scratch.q", 4: f"layer_cache_k.{run}", 5: f"layer_cache_v.{run}"},
              [m.heads, m.kv_heads, m.dim, m.vdim, capacity, M, dtype | m.maps << 8, ldq], [eps])
        _task(t, K_ATTROWS, run, {0: "rows_scratch.q", 1: f"layer_cache_k.{run}", 2: f"layer_cache_v.{run}", 3: "rows_scratch.attention", 4: f"rows_scratch.gate.{i}"},
              [m.heads, m.kv_heads, m.dim, m.vdim, capacity, M, dtype | m.maps << 8, ldq], [m.scale, lambdas[i], m.diff or 0.0, eps])
        linear(run, "rows_scratch.attention", lp + "mix.o", "rows_scratch.y", D, ldo, ld)
        pend, post, top = {1: "rows_scratch.y"}, lp + "norm1b", 0
        if f is None:
            continue
        _task(t, K_RESNORM, run, {0: cur, 2: post, 4: xb, 5: lp + "norm2", 6: h, **pend}, [D, M, dtype, ld, 0, ld], [eps])
        cur, act, lde, lds, lff = xb, 2, round_up(f.experts, 64), round_up(max(f.shared_ff, 1), 64), round_up(f.ff, 64)
        linear(run, h, lp + "mlp.router_shared", "rows_scratch.router", f.experts, ld, lde, f32=1)
        _task(t, K_ROUTE, run, {0: "rows_scratch.router", 1: h, 2: "rows_scratch.chosen_weight", 3: "rows_scratch.chosen", 4: "rows_scratch.rank", 5: "rows_scratch.count",
                                6: "rows_scratch.slot", 7: "rows_scratch.offsets", 8: "rows_scratch.h_grouped"}, [M, f.experts, f.top, lde, ld, dtype])
        linear(run, "rows_scratch.h_grouped", lp + "mlp.experts_up", "rows_scratch.act_grouped", f.ff, ld, lff, act=act, m=M * f.top,
               grouped="rows_scratch.offsets", experts=f.experts)
        linear(run, "rows_scratch.act_grouped", lp + "mlp.experts_down", "rows_scratch.y_grouped", D, lff, ld, m=M * f.top, grouped="rows_scratch.offsets",
               experts=f.experts)
        pend = {8: "rows_scratch.y_grouped", 9: "rows_scratch.slot", 10: "rows_scratch.chosen_weight"}
        if f.shared_ff:
            linear(run, h, lp + "mlp.router_shared", "rows_scratch.shared_act", f.shared_ff, ld, lds, act=act, row0=f.experts)
            linear(run, "rows_scratch.shared_act", lp + "mlp.shared_down", "rows_scratch.y", D, lds, ld)
            pend[1] = "rows_scratch.y"
        post, top = lp + "norm2b", f.top
    if wanted:
        _task(t, K_RESNORM, -1, {0: cur, 2: post, 5: "param.final_norm", 6: "rows_scratch.h_wanted", 7: "rows_scratch.index", **pend},
              [D, wanted, dtype, ld, top, ld], [eps])
        linear(-1, "rows_scratch.h_wanted", "param.lm_head", "rows_scratch.logits", V, ld, V, f32=1, m=wanted)
        if greedy:
            _task(t, K_ARGMAXROW, -1, {0: "rows_scratch.logits"}, [V, M])
    return t


def _pair(a: int, b: int) -> int:
    return a | b << 16


def _limit(layer) -> float:
    return layer.mlp.limit if layer.mlp is not None else 0.0


def _recurrence(layer):
    """The recurrent mixer of a parallel block's layer, the tensors' prefix, the factor on its queries and its gate cap."""
    m = layer.mixer
    if isinstance(m, ParallelMixerSpec):
        return m.right, "mix.right.", 1.0, 0.0
    return m, "mix.", m.dim ** -0.5, m.gate_cap


def _recurrence_bufs(lp: str, pre: str, buf: str, run: int, memory: bool, logits: str, out: str) -> dict:
    bufs = {0: buf + "q", 1: buf + "k", 2: buf + "v", 6: f"layer_state.{run}", 7: out}
    return {**bufs, **({3: logits, 4: lp + pre + "bias"} if memory else {5: lp + pre + "decay"})}


def parallel_decode_tasks(spec, capacity: int, dtype: int = 0, sm: int = 148) -> list:
    """One decoded position of a model of parallel blocks, three or four kernels a layer: the joint projection of everything that
    reads the normed input (the layer before is added up and normed in its prologue, silu and gated unit at its end), attention with
    joint q/k norm, rotation and cache store in its prologue, the recurrence, and the output projections of mixer and feed-forward in
    one launch (the recurrence's norm and gate in its prologue)."""
    D, eps, t = spec.hidden, spec.eps, []
    x = lambda r: f"global_scratch.x_in.{r}"
    _task(t, K_EMBEDROWS, -1, {1: x(0), 3: "param.lm_head"}, [D, 1, spec.vocab])
    cur, pend, post, np_, nn = x(0), None, None, 0, 0
    for run, (i, _) in enumerate(spec.runs()):
        l, lp = spec.layers[i], f"layer_param.{i}."
        m, f, lay, buf = l.mixer, l.mlp, block_layout(l), f"layer_scratch.block.{i}."
        _task(t, K_NORMLIN, run, {0: cur, 1: pend, 2: post, 4: x(run) if run else None, 5: lp + "norm1", 6: lp + "block", 7: "layer_scratch.block", 11: lp + "norm1.b"},
              [D, lay.rows, 3 if lay.silu else 0, 0, np_, nn, lay.exact if f is not None else 0, lay.silu], [eps, 0.5, _limit(l)])
        cur = x(run)
        rec, pre, qs, cap = _recurrence(l)
        both, seg = isinstance(m, ParallelMixerSpec), []
        if both:
            a = m.left
            _task(t, K_WINDEC, run, {0: buf + "attention", 1: lp + "mix.left.q.norm", 2: lp + "mix.left.k.norm", 3: f"layer_cache_k.{run}", 4: f"layer_cache_v.{run}",
                                     5: "layer_scratch.attention", 6: "global_scratch.attention_partials", 7: "global_scratch.attention_counters",
                                     8: f"rotation.{i}" if a.rotary is not None else None},
                  [_pair(a.heads, a.kv_heads), _pair(a.dim, a.vdim), capacity, dtype, key_splits(a, capacity, sm), a.window or 0, a.keep_first, a.rotary.dims if a.rotary else 0],
                  [a.scale, eps])
            seg.append(("layer_scratch.attention", lp + "mix.left.o", a.out_rows))
        _task(t, K_RECDEC, run, _recurrence_bufs(lp, pre, buf, run, not both, buf + "logits", "layer_scratch.memory"), [rec.heads, rec.dim, rec.vdim], [qs, cap])
        seg.append(("layer_scratch.memory", lp + pre + "o", rec.out_rows))
        normed = len(seg) - 1
        if f is not None:
            seg.append((buf + "ff", lp + "mlp.down", f.ff))
        bufs = {6: "layer_scratch.sums", 7: lp + pre + "norm", 8: buf + "gate"}
        for j, (src, w, _) in enumerate(seg):
            bufs[2 * j], bufs[2 * j + 1] = src, w
        ks = [k for _, _, k in seg] + [0] * (3 - len(seg))
        _task(t, K_SEGLIN, run, bufs, [D, len(seg), *ks, normed, rec.norm_group], [eps])
        pend, post, np_, nn = "layer_scratch.sums", lp + "mix.out" if both else None, len(seg), 2 if both else 0
    _task(t, K_NORMLIN, -1, {0: cur, 1: pend, 2: post, 4: x(len(spec.runs())), 5: "param.final_norm", 6: "param.lm_head", 7: "global_scratch.logits",
                             9: "global_scratch.argmax_scratch", 10: "global_scratch.head_counter", 11: "param.final_norm.b"},
          [D, spec.vocab, 0, 0, np_, nn, 0, 0], [eps, 0.5, 0.0, spec.logit_scale])
    return t


def parallel_rows_tasks(spec, capacity: int, rows: int, wanted: int, greedy: bool, dtype: int = 0) -> list:
    """``rows`` consecutive positions of a model of parallel blocks (see layered_rows_tasks)."""
    D, V, M, eps, t = spec.hidden, spec.vocab, rows, spec.eps, []
    ld = round_up(D, 64)
    emb, xb, h, r = "rows_scratch.embedding", "rows_scratch.x", "rows_scratch.h", "rows_scratch."
    _task(t, K_EMBEDROWS, -1, {1: emb, 2: "rows_scratch.tokens", 3: "param.lm_head"}, [D, M, V])
    cur, pend, post, nn = emb, [], None, 0

    def norm(run, w, n, out, x_out=None, index=None):
        _task(t, K_BLOCKNORM, run, {0: cur, **{1 + j: y for j, y in enumerate(pend)}, 4: x_out, 5: w, 6: out, 7: index, 8: w + ".b", 9: post},
              [D, n, dtype, ld, ld, len(pend), nn], [eps, 0.5])

    def linear(run, x, w, y, n, ldx, ldy, f32=0, m=M, scale=0.0):
        _task(t, K_LINROWS, run, {0: x, 1: w, 2: y}, [m, 0, n, ldx, ldy, dtype, f32 << 8, 0], [scale])

    for run, (i, _) in enumerate(spec.runs()):
        l, lp = spec.layers[i], f"layer_param.{i}."
        m, f, lay, buf = l.mixer, l.mlp, block_layout(l), f"rows_scratch.block.{i}."
        norm(run, lp + "norm1", M, h, xb if run else None)
        cur = xb if run else emb
        ldb, ldf, both = round_up(lay.plain, 64), round_up(f.ff, 64) if f is not None else 64, isinstance(m, ParallelMixerSpec)
        _task(t, K_BLOCKLIN, run, {0: h, 1: lp + "block", 2: r + "block", 3: r + "gate_logits" if lay.exact > lay.plain else None, 4: r + "ff" if f is not None else None},
              [M, lay.plain, lay.exact, lay.rows, ldb, ldf, dtype, lay.silu], [_limit(l)])
        pend, post, nn = [], None, 0
        if both:
            a = m.left
            ha, da, lda = _pair(a.heads, a.kv_heads), _pair(a.dim, a.vdim), round_up(a.out_rows, 64)
            _task(t, K_ROTSTORE, run, {0: buf + "attention", 1: lp + "mix.left.q.norm", 2: lp + "mix.left.k.norm", 3: r + "q", 4: f"layer_cache_k.{run}", 5: f"layer_cache_v.{run}",
                                       6: f"rotation.{i}" if a.rotary is not None else None}, [ha, da, capacity, M, ldb, a.rotary.dims if a.rotary else 0, dtype], [eps])
            _task(t, K_WINROWS, run, {0: r + "q", 1: f"layer_cache_k.{run}", 2: f"layer_cache_v.{run}", 3: r + "attention"},
                  [ha, da, capacity, M, dtype, a.window or 0, a.keep_first], [a.scale])
            linear(run, r + "attention", lp + "mix.left.o", r + "y", D, lda, ld)
            pend, post, nn = [r + "y", r + "y1"], lp + "mix.out", 2
        else:
            pend = [r + "y"]
        rec, pre, qs, cap = _recurrence(l)
        ldm, ldg = round_up(rec.out_rows, 8), round_up(rec.out_rows, 64)
        _task(t, K_RECROWS, run, {**_recurrence_bufs(lp, pre, buf, run, not both, r + "gate_logits", r + "memory"), 8: r + "runs"},
              [_pair(rec.heads, dtype), rec.dim, rec.vdim, M, ldb, lay.exact - lay.plain, ldm, recurrence_scratch(rec, M)], [qs, cap])
        _task(t, K_NORMGATE, run, {0: r + "memory", 1: lp + pre + "norm", 2: buf + "gate", 3: r + "gated"}, [rec.out_rows, rec.norm_group, M, ldm, ldb, ldg, dtype], [eps])
        linear(run, r + "gated", lp + pre + "o", pend[-1], D, ldg, ld)
        if f is not None:
            pend.append(r + "y2")
            linear(run, r + "ff", lp + "mlp.down", pend[-1], D, ldf, ld)
    if wanted:
        norm(-1, "param.final_norm", wanted, "rows_scratch.h_wanted", None, "rows_scratch.index")
        linear(-1, "rows_scratch.h_wanted", "param.lm_head", "rows_scratch.logits", V, ld, V, f32=1, m=wanted, scale=spec.logit_scale)
        if greedy:
            _task(t, K_ARGMAXROW, -1, {0: "rows_scratch.logits"}, [V, M])
    return t


def recurrence_cell(rec) -> int:
    """Floats of a recurrence's state per (head, slice of 64 value columns)."""
    return rec.dim * 64 + (round_up(rec.dim + 1, 4) if hasattr(rec, "gate_cap") else 0)


def recurrence_state(rec) -> int:
    return rec.heads * -(-rec.vdim // 64) * recurrence_cell(rec)


def recurrence_scratch(rec, rows: int) -> int:
    """Floats of scratch that let a prompt's chunks be worked on in several runs side by side (at most 16 of at least 4 chunks)."""
    runs = min(16, -(-rows // 64) // 4)
    return 0 if runs < 2 else (runs + 1) * recurrence_state(rec) + runs * rec.heads * -(-rec.vdim // 64)


def emit_layered(spec, capacity: int, lambdas: dict, dtype: int = 0, sm: int = 148) -> dict:
    """The decode step of a layered decoder as a v2 document (``lambdas``: layer -> combination constant of its two maps)."""
    out_slots = {K_EMBEDROWS: [1], K_NORMLIN: [4, 7, 8, 9, 10], K_ATTDEC: [3, 4, 5, 6, 7], K_MOEUP: [3, 4, 5], K_MOEDOWN: [6],
                 K_WINDEC: [3, 4, 5, 6, 7], K_RECDEC: [6, 7], K_SEGLIN: [6]}
    return _envelope(layered_decode_tasks(spec, capacity, lambdas, dtype, sm), out_slots,
                     {"chip": "b200", "arch": "sm_100a", "tensor_parallel": 1, "rank": 0, "bits": 32 if dtype else 16,
                      "launch": "grid and block sizes are chosen by the runtime from the SM count"})


def task_slots(jtask: dict) -> dict:
    """slot -> role of a serialised task (the explicit extra_bindings below slot 100)."""
    return {b["slot"]: b["role"] for b in jtask["extra_bindings"] if b["slot"] < 100}


def write(path, graph: dict):
    """Serialise like the reference does (pretty-printed JSON, task_graph_json.rs:260-270)."""
    import json
    with open(path, "w") as f:
        json.dump(graph, f, indent=2)


def read(path) -> dict:
    import json
    with open(path) as f:
        return json.load(f)


# ------------------------------------------------------------------ lowering a graph the reference wrote
# A task_graph.json written by the reference for a real model names Metal kernels with a fusion-id suffix
# (`fusekit_rmsnorm_qkv_f12`) and carries no shapes: they are constants of the generated shader source.  The per-token list
# it replays has a fixed family order (src/codegen/task_graph_json.rs:1619-1664; python/fusekit_runtime/dispatch.py:3163-3611):
# step_init, embed, per layer [rmsnorm_qkv, sdpa_decode, linear_residual (o_proj), chain (norm -> gate, up -> activation),
# linear_residual (down_proj)], final head, argmax scan / finalize, optional history capture.  Lowering = check that order,
# take the shapes from the model's config.json (checkpoint.spec_from_config), emit this build's graph for them, and say which
# of the reference's parameter roles feed each role of the lowered graph (q|k|v rows concatenated, gate/up paired).
_REF_FAMILIES = ("step_init", "embed_lookup_decode", "rmsnorm_qkv", "sdpa_decode", "linear_residual", "chain", "final_rmsnorm_lm_head",
                 "argmax_logits_scan", "argmax_logits_finalize", "history_capture")
_REF_SKIP = ("step_init", "argmax_logits_scan", "argmax_logits_finalize", "history_capture")     # fused into neighbours here


def reference_family(kernel: str) -> str:
    """`fusekit_<family>[_f<id>][_partial|_combine]` -> family; raises on a kernel this build has no lowering for."""
    import re
    m = re.fullmatch(r"fusekit_([a-z0-9_]+?)(?:_f\d+)?(?:_(?:partial|combine))?", kernel)
    name = m.group(1) if m else ""
    if name not in _REF_FAMILIES:
        raise ValueError(f"no lowering for reference kernel {kernel!r}")
    return name


def lower_reference(doc: dict, spec: ModelSpec, capacity: int, **emit_kw) -> tuple[dict, dict]:
    """Lower a task graph written by the reference (Qwen-shaped default decode list) to this build's graph for `spec`.

    Returns (graph, sources): `graph` is emit(spec, capacity, ...); `sources[role]` lists, in row order, the reference's
    parameter roles (`layer_param.<i>.self_attn.q_proj` ...) whose `weight` / `scales` / `biases` tensors make up that role of
    the lowered graph.  Raises ValueError when the document is not a dispatchable v2 batch-1 graph, when its per-layer kernel
    order is not the one listed above, or when a projection the lowered graph needs is bound nowhere in the layer."""
    if doc.get("version") != VERSION or doc.get("active_m", 1) != 1:
        raise ValueError("reference graph: version 2 and active_m 1 expected")
    if not doc.get("decode_capabilities", {}).get("dispatchable", False):
        raise ValueError("reference graph is not dispatchable")
    if spec.arch != "qwen2":
        raise ValueError("the lowering covers the Qwen-shaped default dispatch list")
    by_id = {t["id"]: t for t in doc["tasks"]}
    per_layer: dict[int, list] = {}
    head_seen = embed_seen = False
    for tid in doc["decode_pipeline"]:
        t = by_id[tid]
        fam = reference_family(t["kernel"])
        if fam in _REF_SKIP:
            continue
        if fam == "embed_lookup_decode":
            embed_seen = True
        elif fam == "final_rmsnorm_lm_head":
            head_seen = True
        else:
            if "layer_idx" not in t:
                raise ValueError(f"reference task {tid} ({t['kernel']}) carries no layer_idx")
            fams = per_layer.setdefault(int(t["layer_idx"]), [])
            if not (fam == "sdpa_decode" and fams and fams[-1][0] == "sdpa_decode"):      # partial + combine count once
                fams.append((fam, t))
    if not embed_seen or not head_seen:
        raise ValueError("reference graph lacks the embed lookup or the final head")
    if sorted(per_layer) != list(range(spec.n_layers)):
        raise ValueError(f"reference graph has layers {sorted(per_layer)[:3]}..., the model {spec.n_layers}")
    want = ["rmsnorm_qkv", "sdpa_decode", "linear_residual", "chain", "linear_residual"]
    sources: dict[str, list] = {"param.embed_tokens": ["param.embed_tokens"], "param.final_norm": ["param.final_norm"], "param.lm_head": ["param.lm_head"]}
    for l in range(spec.n_layers):
        got = [f for f, _ in per_layer[l]]
        if got != want:
            raise ValueError(f"layer {l}: kernel order {got}, expected {want}")
        bound = set()
        for _, t in per_layer[l]:
            for b in list(t.get("extra_bindings", [])) + [{"role": x.get("role_name", "")} for x in t.get("inputs", [])]:
                r = b.get("role", "")
                if r.startswith(f"layer_param.{l}."):
                    rel = r[len(f"layer_param.{l}."):]
                    for suffix in (".weight", ".scales", ".biases", ".bias"):
                        if rel.endswith(suffix):
                            rel = rel[: -len(suffix)]
                            break
                    bound.add(rel)
        need = ["self_attn.q_proj", "self_attn.k_proj", "self_attn.v_proj", "self_attn.o_proj", "mlp.gate_proj", "mlp.up_proj", "mlp.down_proj"]
        missing = [n for n in need if n not in bound]
        if missing:
            raise ValueError(f"layer {l}: the reference graph binds no {missing}")
        lp = f"layer_param.{l}."
        sources[lp + "self_attn.qkv_proj"] = [lp + "self_attn.q_proj", lp + "self_attn.k_proj", lp + "self_attn.v_proj"]
        sources[lp + "self_attn.qkv_proj.bias"] = [lp + "self_attn.q_proj.bias", lp + "self_attn.k_proj.bias", lp + "self_attn.v_proj.bias"]
        sources[lp + "self_attn.o_proj"] = [lp + "self_attn.o_proj"]
        sources[lp + "mlp.gate_up_proj"] = [lp + "mlp.gate_proj", lp + "mlp.up_proj"]
        sources[lp + "mlp.down_proj"] = [lp + "mlp.down_proj"]
        sources[lp + "input_layernorm.weight"] = [lp + "input_layernorm.weight"]
        sources[lp + "post_attention_layernorm.weight"] = [lp + "post_attention_layernorm.weight"]
    return emit(spec, capacity, **emit_kw), sources
