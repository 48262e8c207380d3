"""Layers of a hybrid design beside Qwen2 layers of equal width: `python bench.py --model bazirax-0.5b` or
`lozanex-0.5b` (also -1.5b, -7b).

Both models have the same width, feed-forward (of a mixture of experts: what a token uses of it), head count
and size, layer count and vocabulary, random bf16 weights; decode is a captured step of `--batch` sequences at
`--context` tokens, prefill whole prompts. Then every kernel of the new layers alone, over copies of its data
that together exceed L2, against the measured copy bandwidth and GEMM throughput, with the like kernels of
the existing layers. CUDA events throughout."""

from __future__ import annotations

import json
import statistics
from pathlib import Path

import torch

SIZES = {
    "bazirax-0.5b": dict(width=896, ff=4864, heads=14, dim=64, kv_heads=2, q_rank=448, kv_rank=256),
    "bazirax-1.5b": dict(width=2048, ff=8192, heads=16, dim=128, kv_heads=2, q_rank=768, kv_rank=512),
    "bazirax-7b": dict(width=3584, ff=18944, heads=28, dim=128, kv_heads=4, q_rank=1536, kv_rank=512),
}
# `active` of `experts` experts and a shared one per token, which together are as wide as the dense feed-forward
EXPERTS = {"0.5b": dict(experts=16, active=2), "1.5b": dict(experts=32, active=4), "7b": dict(experts=32, active=4)}
for _name, _experts in EXPERTS.items():
    SIZES["lozanex-" + _name] = {**SIZES["bazirax-" + _name], **_experts}
VOCAB = 32768
PEAKS = Path(__file__).resolve().parent / "MEASURED_PEAKS.json"


def bazirax_config(size):
    from llm_compiler_b200 import bazirax

    heads, dim = size["heads"], size["dim"]
    delta = dict(heads=heads, kv_heads=heads, dim=dim, vdim=dim, conv=4)
    retention = dict(heads=heads, dim=dim, vdim=dim, rot=dict(base=1e4, dims=dim),
                     decay=[1 - 2.0 ** -(5 + i * 5 / heads) for i in range(heads)])
    latent = dict(heads=heads, dim=dim, vdim=dim, q_rank=size["q_rank"], kv_rank=size["kv_rank"], scale=dim ** -0.5)
    kinds = [("channel_delta", delta), ("retention", retention), ("latent_attention", latent)]
    layers = [bazirax.LayerSpec(kind, spec, size["ff"]) for kind, spec in kinds * 2]
    layers[5] = bazirax.LayerSpec("latent_attention", dict(latent, kv_from=2), size["ff"])
    return bazirax.BaziraxConfig(vocab_size=VOCAB, hidden_size=size["width"], norm_eps=1e-5, layers=tuple(layers))


def lozanex_config(size):
    from llm_compiler_b200 import lozanex

    heads, dim = size["heads"], size["dim"]
    delta = dict(heads=heads, kv_heads=heads, dim=dim, vdim=dim, conv=4)
    attention = dict(heads=heads, kv_heads=size["kv_heads"], dim=dim, vdim=dim, scale=dim ** -0.5,
                     rot=dict(base=1e6, dims=dim), mask=dict(size=8192))
    mlp = dict(kind="moe", expert=dict(ff=size["ff"] // 2 // size["active"]),
               router=dict(experts=size["experts"], top=size["active"]), shared=dict(ff=size["ff"] // 2))
    layers = [lozanex.LayerSpec(*spec, mlp) for spec in (
        ("delta", delta), ("attention", attention), ("delta", delta), ("delta", delta),
        ("attention", dict(attention, kv_from=1)), ("delta", delta))]
    return lozanex.LozanexConfig(vocab_size=VOCAB, hidden_size=size["width"], norm_eps=1e-5, layers=tuple(layers))


def qwen_config(size, layers):
    from llm_compiler_b200 import qwen2

    return qwen2.Qwen2Config(hidden_size=size["width"], intermediate_size=size["ff"], num_layers=layers,
                             num_heads=size["heads"], num_kv_heads=size["kv_heads"], rope_theta=1e6,
                             vocab_size=VOCAB, head_dim_override=size["dim"])


def milliseconds(call, repeats=10, warmup=3):
    for _ in range(warmup):
        call()
    torch.cuda.synchronize()
    times = []
    for _ in range(repeats):
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        begin.record()
        call()
        end.record()
        end.synchronize()
        times.append(begin.elapsed_time(end))
    return statistics.median(times)


def graph_milliseconds(calls, rounds=1):
    """One launch's time: all calls (each on data of its own) in one graph."""
    for call in calls:
        call()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for _ in range(rounds):
            for call in calls:
                call()
    return milliseconds(graph.replay) / (rounds * len(calls))


def decode_ms(engine, context, batch):
    lengths = [context] * batch
    engine.load_context(torch.tensor(lengths))
    engine.input_ids.copy_(torch.randint(0, VOCAB, (batch,)))
    engine.capture()

    def steps():
        for _ in range(20):
            engine._graph.replay()

    time = milliseconds(steps, repeats=5, warmup=1) / 20
    engine.load_context(torch.tensor(lengths))
    return time


def bazirax_kernels(engine, config, size, context, batch, hbm_gbs, tflops):
    """Every kernel of the hybrid layers alone. bytes: what must cross HBM; flops: matrix products."""
    from llm_compiler_b200 import hybrid_kernels as hk, kernels

    rows = {}

    def record(name, calls, nbytes=0, flops=0):
        ms = graph_milliseconds(calls)
        floor = max(nbytes / (hbm_gbs * 1e6), flops / (tflops * 1e9))
        rows[name] = {"us": round(ms * 1e3, 2), "of_roofline": round(floor / ms, 3),
                      "bound": "memory" if nbytes / (hbm_gbs * 1e6) >= flops / (tflops * 1e9) else "tensor"}

    device = engine.device
    heads, dim, width, rank = size["heads"], size["dim"], size["width"], size["kv_rank"]
    delta, retention, latent = (engine.layers[i].mixer for i in range(3))
    rand = lambda *shape: torch.randn(*shape, device=device)
    bf16 = lambda *shape: (0.5 * rand(*shape)).to(torch.bfloat16)
    vector = lambda values: torch.tensor(values, dtype=torch.int32, device=device)

    # ---- decode, `batch` sequences ----
    step = hk.SequenceBatch(batch, batch, vector(range(batch)), vector(range(batch + 1)), vector(range(batch)),
                            vector([context] * batch))
    copies = max(2, int(3e8 / (batch * heads * dim * dim * 4)))
    states = [0.1 * rand(batch, heads, dim, dim) for _ in range(copies)]
    state_bytes = batch * heads * (2 * dim * dim * 4 + 5 * dim * 2)
    projected, gates = bf16(batch, delta.w_in.shape[0]), bf16(batch, delta.w_gates.shape[0])
    ring = bf16(batch, delta.taps, 3 * heads * dim)
    inputs = hk.delta_inputs(projected, gates, delta.conv, delta.a_log, delta.dt_bias, ring, step, heads=heads,
                             kv_heads=heads, dim=dim, vdim=dim, columns=delta.columns,
                             decay_column=delta.decay_column, q_scale=delta.q_scale)
    gate = gates[:, delta.gate_column:]
    record("decode: delta step", [lambda s=s: hk.recurrence_step(inputs, s, gate, delta.norm, batch, kind="sigmoid",
                                                                epsilon=1e-5) for s in states], state_bytes)
    plain = bf16(batch, retention.w_in.shape[0])
    r_inputs = hk.retention_inputs(plain, retention.decay, step, heads=heads, dim=dim, vdim=dim,
                                   columns=retention.columns, rot_dims=dim, rot_base=1e4, k_scale=1.0)
    r_gate = plain[:, retention.gate_column:]
    record("decode: retention step", [lambda s=s: hk.recurrence_step(r_inputs, s, r_gate, None, batch, kind="silu",
                                                                    epsilon=1e-5) for s in states], state_bytes)
    del states
    caches = [bf16(batch, context + 64, latent.rank_row) for _ in range(max(2, int(3e8 / (batch * context * rank * 2))))]
    absorbed = bf16(batch, heads, latent.rank_row)
    record("decode: latent attention", [lambda c=c: hk.latent_attention(absorbed, c, latent.sink, step, scale=0.1)
                                        for c in caches], batch * (context + 1) * rank * 2, 4 * batch * heads * context * rank)
    del caches
    q = bf16(batch, heads, latent.q_size)
    weights = [bf16(*latent.w_into.shape) for _ in range(max(2, int(2e8 / latent.w_into.numel() / 2)))]
    record("decode: into the latent space", [lambda w=w: hk.head_linear(q, w) for w in weights],
           weights[0].numel() * 2 + absorbed.numel() * 2)
    parts, norm = rand(4, batch, width), bf16(width)
    x = rand(batch, width)
    record("decode: residual norm", [lambda: hk.residual_norm(x, parts, norm, norm, epsilon=1e-5, weight_offset=1.0,
                                                              dtype=torch.bfloat16)] * 8, batch * width * (16 + 8 + 2))

    # ---- one prompt of 4096 tokens, and four ----
    for sequences in (1, 4):
        tokens = 4096
        n = sequences * tokens
        name = f"prefill {sequences} x {tokens}: "
        slots = list(range(sequences))
        prompt = hk.SequenceBatch(n, sequences, vector([i for i in slots for _ in range(tokens)]),
                                  vector([i * tokens for i in range(sequences + 1)]), vector(slots),
                                  vector([0] * sequences), [tokens] * sequences, [0] * sequences, slots)
        prompt.chunk_table()
        big, big_gates = bf16(n, delta.w_in.shape[0]), bf16(n, delta.w_gates.shape[0])
        inputs = hk.delta_inputs(big, big_gates, delta.conv, delta.a_log, delta.dt_bias, ring, prompt, heads=heads,
                                 kv_heads=heads, dim=dim, vdim=dim, columns=delta.columns,
                                 decay_column=delta.decay_column, q_scale=delta.q_scale)
        operands = hk.delta_prep(inputs, prompt, torch.bfloat16, device)
        state = 0.1 * rand(sequences, heads, dim, dim)
        unit = n * heads * dim
        # necessary traffic: the bf16 projections once and the gated result once
        chunk_flops = 2 * n * heads * (64 * dim * 3 + 3 * dim * dim)

        def delta_core():
            o = hk.delta_prep(inputs, prompt, torch.bfloat16, device)
            out = hk.recurrence(*o, state, prompt, torch.bfloat16)
            hk.gated_head_norm(out, delta.norm, big_gates[:, delta.gate_column:], kind="sigmoid", epsilon=1e-5)

        record(name + "delta rule, all launches", [delta_core], unit * 2 * 6, chunk_flops)
        record(name + "delta prep", [lambda: hk.delta_prep(inputs, prompt, torch.bfloat16, device)], unit * (8 + 16))
        record(name + "delta chunks", [lambda: hk.recurrence(*operands, state, prompt, torch.bfloat16)],
               unit * (16 + 4), chunk_flops)
        read_out = rand(n, heads, dim)
        record(name + "gated head norm", [lambda: hk.gated_head_norm(read_out, delta.norm, big_gates[:, delta.gate_column:],
                                                                     kind="sigmoid", epsilon=1e-5)], unit * 8)
        del operands
        big = bf16(n, retention.w_in.shape[0])
        r_inputs = hk.retention_inputs(big, retention.decay, prompt, heads=heads, dim=dim, vdim=dim,
                                       columns=retention.columns, rot_dims=dim, rot_base=1e4, k_scale=1.0)

        def retention_core():
            q, k, v = hk.retention_prep(r_inputs, n, torch.bfloat16, device)
            out = hk.recurrence(q, k, v, None, retention.decay, state, prompt, torch.bfloat16)
            hk.gated_head_norm(out, None, big[:, retention.gate_column:], kind="silu", epsilon=1e-5)

        record(name + "retention, all launches", [retention_core], unit * 2 * 5,
               2 * n * heads * (64 * dim * 2 + 2 * dim * dim))
        q = bf16(sequences, tokens, heads, latent.q_size)
        kv = bf16(sequences, tokens, 2 * heads, latent.q_size)
        out = torch.empty_like(q)
        record(name + "attention", [lambda: hk.context_attention(
            q.transpose(1, 2), kv[:, :, :heads].transpose(1, 2), kv[:, :, heads:].transpose(1, 2), latent.sink, out,
            context=0, scale=0.1)], 0, 2 * sequences * heads * tokens * tokens * dim)
        record(name + "attention, Qwen2's call", [lambda: kernels.b200_prefill_attention(
            q.transpose(1, 2), kv[:, :, :heads].transpose(1, 2), kv[:, :, heads:].transpose(1, 2), None, scale=0.1,
            causal=True)], 0, 2 * sequences * heads * tokens * tokens * dim)
        x, y = rand(n, width), bf16(n, width)
        record(name + "residual norm", [lambda: hk.residual_norm(x, y, norm, norm, epsilon=1e-5, weight_offset=1.0,
                                                                 dtype=torch.bfloat16)], n * width * 12)
        h = bf16(n, width)
        record(name + "RMS norm, Qwen2's", [lambda: kernels.b200_rms_norm(h, norm, epsilon=1e-5)], n * width * 4)
    return rows


def lozanex_kernels(engine, config, size, context, batch, hbm_gbs, tflops):
    """Every kernel of the Lozanex layers alone, and the like kernels of Bazirax and Qwen2 layers on the same
    shapes. bytes: what must cross HBM; flops: matrix products."""
    from llm_compiler_b200 import hybrid_kernels as hk, kernels

    rows = {}

    def record(name, calls, nbytes=0, flops=0):
        ms = graph_milliseconds(calls)
        floor = max(nbytes / (hbm_gbs * 1e6), flops / (tflops * 1e9))
        rows[name] = {"us": round(ms * 1e3, 2), "of_roofline": round(floor / ms, 3),
                      "bound": "memory" if nbytes / (hbm_gbs * 1e6) >= flops / (tflops * 1e9) else "tensor"}

    device = engine.device
    heads, kv_heads, dim, width = size["heads"], size["kv_heads"], size["dim"], size["width"]
    delta, attention, mlp = engine.layers[0].mixer, engine.layers[1].mixer, engine.layers[0].mlp
    experts, top = size["experts"], size["active"]
    ff, shared_ff = mlp.w_out.shape[2], mlp.shared.w_out.shape[1]
    rand = lambda *shape: torch.randn(*shape, device=device)
    bf16 = lambda *shape: (0.5 * rand(*shape)).to(torch.bfloat16)
    vector = lambda values: torch.tensor(values, dtype=torch.int32, device=device)
    copies_of = lambda nbytes: max(2, int(3e8 / nbytes))

    def delta_block(projected, ring, part):
        return hk.delta_inputs(projected, projected, delta.conv, delta.a_log, delta.dt_bias, ring, part, heads=heads,
                               kv_heads=heads, dim=dim, vdim=dim, columns=delta.columns,
                               decay_column=delta.decay_column, q_scale=delta.q_scale)

    def prepare(projected, bias, keys, values, part):
        return hk.attention_prep(projected, bias, attention.q_norm, attention.k_norm, attention.turns, keys, values, part,
                                 heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, row_size=dim,
                                 columns=attention.columns, epsilon=1e-5)

    def expert_rows(name, n):
        """The mixture of experts on n rows, launch by launch, and dense projections of the same size."""
        h = bf16(n, width)
        few, tile = n <= 128, mlp.tile_of(n)
        always = mlp.slices if few else 0  # the shared expert in slices
        used, each = min(experts, n * top) + always, top + always
        weight_sets = copies_of(mlp.w_in.numel() * 2)
        w_in = [mlp.w_in] + [mlp.w_in.clone() for _ in range(weight_sets - 1)]
        w_out = [mlp.w_out] + [mlp.w_out.clone() for _ in range(weight_sets - 1)]
        if few:
            choose = lambda: hk.expert_select(h, mlp.w_router, mlp.counters, top=top, always=always, tile=tile)
            record(name + "choice of experts", [choose] * 8, (h.numel() + mlp.w_router.numel()) * 2)
        else:
            logits = kernels.b200_linear_partial(h, mlp.w_router)
            choose = lambda: hk.expert_route(logits, h, mlp.counters, top=top, always=0, tile=tile)
            record(name + "router logits", [lambda: kernels.b200_linear_partial(h, mlp.w_router)] * 8,
                   (h.numel() + mlp.w_router.numel()) * 2 + n * mlp.w_router.shape[0] * 4, 2 * n * mlp.w_router.numel())
            record(name + "choice of experts, rows in order", [choose] * 8, logits.numel() * 4 + h.numel() * 2 * (1 + top))
        order, ordered = (choose(), h) if few else choose()
        inner = hk.grouped_linear(ordered, mlp.w_in, order, gather=few, swiglu=True)
        record(name + "experts, gate and up", [lambda w=w: hk.grouped_linear(ordered, w, order, gather=few, swiglu=True)
                                               for w in w_in],
               (used * 2 * ff * width + n * width + n * each * ff) * 2, 4 * n * each * ff * width)
        record(name + "experts, down", [lambda w=w: hk.grouped_linear(inner, w, order) for w in w_out],
               (used * ff * width + n * each * (width + ff)) * 2, 2 * n * each * ff * width)
        dense = bf16(top * n, width)
        sets = copies_of(4 * ff * width)
        w_dense = [bf16(2 * ff, width) for _ in range(sets)]
        record(name + f"dense gate and up, {top * n} rows (Qwen2's)",
               [lambda w=w: kernels.b200_linear(dense, w, epilogue="swiglu") for w in w_dense],
               (2 * ff * width + n * top * (width + ff)) * 2, 4 * n * top * ff * width)
        w_down = [bf16(width, ff) for _ in range(sets)]
        dense = bf16(top * n, ff)
        record(name + f"dense down, {top * n} rows (Qwen2's)", [lambda w=w: kernels.b200_linear(dense, w) for w in w_down],
               (ff * width + n * top * (width + ff)) * 2, 2 * n * top * ff * width)
        x, norm = rand(n, width), bf16(width)
        y = hk.Summands(None if few else bf16(n, width), None, hk.grouped_linear(inner, mlp.w_out, order), order.places)
        record(name + "residual norm over experts", [lambda: hk.residual_norm(
            x, y, norm, None, epsilon=1e-5, weight_offset=0.0, dtype=torch.bfloat16, narrow=True)] * 8,
            n * width * (8 + 2 + 2 * each + (0 if few else 2)))

    # ---- decode, `batch` sequences ----
    step = hk.SequenceBatch(batch, batch, vector(range(batch)), vector(range(batch + 1)), vector(range(batch)),
                            vector([context] * batch))
    states = [0.1 * rand(batch, heads, dim, dim) for _ in range(copies_of(batch * heads * dim * dim * 4))]
    projected, ring = bf16(batch, delta.w_in.shape[0]), bf16(batch, delta.taps, 3 * heads * dim)
    inputs, gate = delta_block(projected, ring, step), projected[:, delta.gate_column:]
    record("decode: delta step", [lambda s=s: hk.recurrence_step(inputs, s, gate, delta.norm, batch, kind="silu", epsilon=1e-5)
                                  for s in states], batch * heads * (2 * dim * dim * 4 + 5 * dim * 2))
    gates = bf16(batch, 2 * heads * dim)
    channel = hk.delta_inputs(projected, gates, delta.conv, delta.a_log, bf16(heads * dim), ring, step, heads=heads,
                              kv_heads=heads, dim=dim, vdim=dim, columns=delta.columns, decay_column=0, q_scale=delta.q_scale)
    record("decode: delta step (Bazirax's)", [lambda s=s: hk.recurrence_step(
        channel, s, gates[:, heads * dim:], delta.norm, batch, kind="sigmoid", epsilon=1e-5) for s in states],
        batch * heads * (2 * dim * dim * 4 + 5 * dim * 2))
    del states
    cache_bytes = 2 * batch * context * kv_heads * dim * 2
    caches = [(bf16(batch, context + 64, kv_heads, dim), bf16(batch, context + 64, kv_heads, dim))
              for _ in range(copies_of(cache_bytes))]
    parts = rand(4, batch, attention.w_in.shape[0])
    record("decode: attention prep", [lambda c=c: prepare(parts, attention.bias, *c, step) for c in caches],
           parts.numel() * 4 + batch * (heads + 2 * kv_heads) * dim * 2)
    q = bf16(batch, heads, dim)
    record("decode: attention", [lambda c=c: hk.slot_decode_attention(q, *c, step, scale=0.1, chunk=8192) for c in caches],
           cache_bytes)
    record("decode: attention, chunks of 1024", [lambda c=c: hk.slot_decode_attention(
        q, *c, hk.SequenceBatch(batch, batch, step.token_sequence, step.starts, step.slots, late), scale=0.1, chunk=1024)
        for late in (vector([context - 1] * batch),) for c in caches], cache_bytes // context * 1024)
    lengths = torch.full((batch,), context + 1, dtype=torch.int64, device=device)
    record("decode: attention (Qwen2's)", [lambda c=c: kernels.b200_decode_attention(
        q.view(batch, heads, 1, dim), *c, lengths, None, scale=0.1) for c in caches], cache_bytes)
    del caches
    expert_rows("decode: ", batch)

    # ---- one prompt of 4096 tokens, and four ----
    for sequences in (1, 4):
        tokens = 4096
        n = sequences * tokens
        name = f"prefill {sequences} x {tokens}: "
        slots = list(range(sequences))
        prompt = hk.SequenceBatch(n, sequences, vector([i for i in slots for _ in range(tokens)]),
                                  vector([i * tokens for i in range(sequences + 1)]), vector(slots),
                                  vector([0] * sequences), [tokens] * sequences, [0] * sequences, slots)
        prompt.chunk_table()
        big = bf16(n, delta.w_in.shape[0])
        inputs = delta_block(big, ring, prompt)
        state = 0.1 * rand(sequences, heads, dim, dim)
        unit = n * heads * dim
        chunk_flops = 2 * n * heads * (64 * dim * 3 + 3 * dim * dim)

        def delta_core():
            o = hk.delta_prep(inputs, prompt, torch.bfloat16, device)
            out = hk.recurrence(*o, state, prompt, torch.bfloat16)
            hk.gated_head_norm(out, delta.norm, big[:, delta.gate_column:], kind="silu", epsilon=1e-5)

        record(name + "delta rule, all launches", [delta_core], unit * 2 * 5, chunk_flops)
        operands = hk.delta_prep(inputs, prompt, torch.bfloat16, device)
        record(name + "delta prep", [lambda: hk.delta_prep(inputs, prompt, torch.bfloat16, device)], unit * (6 + 12))
        record(name + "delta chunks", [lambda: hk.recurrence(*operands, state, prompt, torch.bfloat16)],
               unit * (12 + 4), chunk_flops)
        per_channel = (*operands[:4], operands[4].expand(-1, -1, dim).contiguous())
        record(name + "delta chunks (Bazirax's)", [lambda: hk.recurrence(*per_channel, state, prompt, torch.bfloat16)],
               unit * (16 + 4), chunk_flops)
        del operands, per_channel, big
        keys, values = bf16(sequences, tokens, kv_heads, dim), bf16(sequences, tokens, kv_heads, dim)
        big = bf16(n, attention.w_in.shape[0])
        record(name + "attention prep", [lambda: prepare(big, None, keys, values, prompt)],
               n * 2 * (heads + 2 * kv_heads) * dim * 2)
        q = bf16(sequences, tokens, heads, dim)
        out = torch.empty_like(q)
        attend = lambda chunk: hk.context_attention(q.transpose(1, 2), keys.transpose(1, 2), values.transpose(1, 2), None,
                                                    out, context=0, scale=0.1, chunk=chunk)
        flops = 2 * sequences * heads * tokens * dim
        record(name + "attention", [lambda: attend(8192)], 0, flops * tokens)
        record(name + "attention, chunks of 1024", [lambda: attend(1024)], 0, flops * 1024)
        record(name + "attention (Qwen2's)", [lambda: kernels.b200_prefill_attention(
            q.transpose(1, 2), keys.transpose(1, 2), values.transpose(1, 2), None, scale=0.1, causal=True)], 0, flops * tokens)
        expert_rows(name, n)
        h, norm = bf16(n, width), bf16(width)
        record(name + "RMS norm (Qwen2's)", [lambda: kernels.b200_rms_norm(h, norm, epsilon=1e-5)], n * width * 4)
    return rows


def run(args, hbm_gbs):
    from llm_compiler_b200 import bazirax, lozanex, qwen2
    from llm_compiler_b200.engine import Qwen2Engine
    from llm_compiler_b200.hybrid_engine import HybridEngine

    torch.manual_seed(0)
    size = SIZES[args.model]
    design = args.model.split("-")[0]
    module, make_config, kernel_table = {"bazirax": (bazirax, bazirax_config, bazirax_kernels),
                                         "lozanex": (lozanex, lozanex_config, lozanex_kernels)}[design]
    config = make_config(size)
    other = qwen_config(size, config.num_layers)
    batch, context = args.batch, args.context
    peaks = json.loads(PEAKS.read_text()) if PEAKS.exists() else {}
    tflops = peaks.get("bf16_tflops", 1590.0)
    result = {}
    engines = {
        design: lambda b, c: HybridEngine(config, weights, batch=b, capacity=c),
        "qwen2": lambda b, c: Qwen2Engine(other, weights, batch=b, capacity=c),
    }
    for name, build in engines.items():
        if name == design:
            more = dict(gate_rank=size["dim"]) if design == "bazirax" else {}
            weights = module.make_weights(config, dtype=torch.bfloat16, device="cuda", **more)
        else:
            weights = qwen2.make_weights(other, dtype=torch.bfloat16, device="cuda", reproducible=False)
        entry = result[name] = {"parameters": sum(w.numel() for w in weights.values())}
        for sequences, tokens in ((1, 4096), (4, 4096), (16, 512)):
            engine = build(sequences, tokens + 64)
            ids = torch.randint(0, VOCAB, (sequences, tokens))
            ms = milliseconds(lambda: engine.prefill(ids), repeats=5)
            entry[f"prefill {sequences} x {tokens}"] = {"ms": round(ms, 3), "tokens_per_s": round(sequences * tokens / ms * 1e3)}
            del engine
        engine = build(batch, context + 512)
        ms = decode_ms(engine, context, batch)
        entry[f"decode {batch} x {context}"] = {"ms": round(ms, 4), "tokens_per_s": round(batch / ms * 1e3),
                                                "kernels": engine.kernels_per_step}
        if name == design:
            entry["kernels"] = kernel_table(engine, config, size, context, batch, hbm_gbs, tflops)
        del engine, weights
        torch.cuda.empty_cache()
    decode = result[design][f"decode {batch} x {context}"]
    return {"metric": f"{args.model}_layers_decode_tokens_per_s", "value": decode["tokens_per_s"], "unit": "tokens/s",
            "n_gpus": 1, "ms_per_step": decode["ms"], "higher_is_better": True, "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic", "config": {"model": args.model, "layers": config.num_layers, "vocab": VOCAB,
                                            "batch": batch, "context": context, "peaks": {"hbm_gbs": hbm_gbs, "bf16_tflops": tflops},
                                            "l2": "kernel rows rotate over copies larger than L2"},
            "results": result}
