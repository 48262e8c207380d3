"""Hybrid layers on the GPU against the plain implementation of oracle/hybrid_model.py: every mechanism
alone, prompts in portions of any size against whole prompts and token-by-token decoding, unequal batches
against each sequence alone, slots that are used again, and greedy generation through the scheduler.

fp32 runs are compared tightly; bf16 runs (16-bit projections, fp32 recurrences, scores and norms) within
a few rounding errors of the same bf16 weights in double precision.
"""

import io
import json

import numpy as np
import pytest
import torch

from llm_compiler_b200 import bazirax, kernels
from llm_compiler_b200 import hybrid_kernels as hk
from llm_compiler_b200.cli import main
from llm_compiler_b200.hybrid_engine import HybridEngine
from llm_compiler_b200.kv_state import ExecutionError
from llm_compiler_b200.mixers import ChannelDelta, LatentAttention, Retention
from llm_compiler_b200.registry import load_model
from llm_compiler_b200.safetensors_io import save_safetensors
from llm_compiler_b200.scheduler import RequestScheduler
from llm_compiler_b200.trace import replay
from hybrid_helpers import (BOTH, CUTS, EPS, MODEL_TOLERANCE, TOLERANCE, batch_of, close, cuda, double, random_rows,
                            run_cut, run_mixer, tokens_of)
from oracle import hybrid_model as oracle

pytestmark = pytest.mark.gpu


def mixer_weights(kind, spec, width, dtype, *, gate_rank=12, seed=0):
    config = bazirax.BaziraxConfig(vocab_size=8, hidden_size=width, norm_eps=EPS,
                                   layers=(bazirax.LayerSpec(kind, spec, None),))
    weights = bazirax.make_weights(config, seed=seed, dtype=dtype, gate_rank=gate_rank)
    return {name[len("l0.mix."):]: w for name, w in weights.items() if name.startswith("l0.mix.")}


# ------------------------------------------------------------------------------ norms ----
@BOTH
@pytest.mark.parametrize("width", [48, 52, 1000])
def test_residual_norm(dtype, width):
    g = torch.Generator().manual_seed(width)
    x = torch.randn(5, width, generator=g)
    y = torch.randn(5, hk.pad8(width), generator=g).to(dtype)
    post, after = (0.2 * torch.randn(2, width, generator=g)).to(dtype)
    want = x.double() + oracle.rms_norm(y[:, :width].double(), post.double(), EPS, 1.0)
    residual = x.cuda()
    h = hk.residual_norm(residual, y.cuda(), post.cuda(), after.cuda(), epsilon=EPS, weight_offset=1.0, dtype=dtype)
    assert float((residual.double().cpu() - want).abs().max()) < 1e-5  # the residual stays fp32
    assert torch.all(h[:, width:] == 0)
    close(h[:, :width], oracle.rms_norm(want, after.double(), EPS, 1.0), dtype)
    parts = torch.randn(3, 5, width, generator=g)
    residual = x.cuda()
    assert hk.residual_norm(residual, parts.cuda(), post.cuda(), None, epsilon=EPS, weight_offset=0.0,
                            dtype=dtype) is None
    want = x.double() + oracle.rms_norm(parts.double().sum(0), post.double(), EPS)
    assert float((residual.double().cpu() - want).abs().max()) < 1e-5


@BOTH
@pytest.mark.parametrize("width", [36, 50])
def test_embedding_residual(dtype, width):
    table = torch.randn(11, width, generator=torch.Generator().manual_seed(0)).to(dtype).cuda()
    ids = torch.tensor([3, 0, 10, 3], device="cuda")
    assert torch.equal(hk.embedding_residual(table, ids), table.float()[ids])
    kernels.runtime().check_status()
    x = hk.embedding_residual(table, torch.tensor([11, 2], device="cuda"))
    with pytest.raises(kernels.KernelStatusError, match="token id"):
        kernels.runtime().check_status()
    assert torch.all(x[0] == 0) and torch.equal(x[1], table.float()[2])


# -------------------------------------------------------------------------- retention ----
RETENTION = [
    dict(heads=3, dim=24, vdim=40, rot=dict(base=1e4, dims=16), decay=[0.5, 0.97, 0.9999]),
    dict(heads=2, dim=64, vdim=64, rot=dict(base=1e6, dims=64), decay=[0.96, 0.999]),
    dict(heads=1, dim=128, vdim=48, rot=dict(base=500.0, dims=32), decay=[0.99]),
    dict(heads=2, dim=20, vdim=9, rot=dict(base=1e4, dims=0), decay=[1.0, 0.1]),
    dict(heads=2, dim=128, vdim=128, rot=dict(base=1e4, dims=128), decay=[0.98, 0.9995]),
]


def retention_mixer(spec, weights, width):
    return Retention(cuda(weights), width=width, heads=spec["heads"], dim=spec["dim"], vdim=spec["vdim"],
                     decay=spec["decay"], rot_dims=spec["rot"]["dims"], rot_base=spec["rot"]["base"], epsilon=EPS)


@BOTH
@pytest.mark.parametrize("index", range(len(RETENTION)))
def test_retention(dtype, index):
    spec, width = RETENTION[index], [40, 64, 36, 72, 128][index]
    weights = mixer_weights("retention", spec, width, dtype, seed=index)
    h = random_rows(150, width, dtype, 10 + index)
    want = oracle.retention(double(weights), spec, h.double(), EPS)
    mixer = retention_mixer(spec, weights, width)
    for cuts in CUTS:
        close(run_mixer(mixer, h, cuts), want, dtype)


def test_rotation_far_from_the_start():
    """A portion at a far position turns by the exact angle: q and k of one token keep their product,
    and two tokens' product depends on their distance only."""
    weights = mixer_weights("retention", RETENTION[1], 64, torch.float32)
    h = random_rows(4, 64, torch.float32, 3)
    mixer = retention_mixer(RETENTION[1], weights, 64)
    pieces = []
    for base in (0, 100000):
        projected = kernels.b200_linear(h.cuda(), mixer.w_in)
        inputs = hk.retention_inputs(projected, mixer.decay, batch_of([(0, base, 4)]), heads=2, dim=64, vdim=64,
                                     columns=mixer.columns, rot_dims=64, rot_base=1e6, k_scale=mixer.k_scale)
        q, k, _ = hk.retention_prep(inputs, 4, torch.float32, h.cuda().device)
        pieces.append(torch.einsum("ihd,jhd->hij", q.double(), k.double()))
    assert float((pieces[0] - pieces[1]).abs().max()) < 1e-5 * float(pieces[0].abs().max())


# ------------------------------------------------------------------------- delta rule ----
DELTA = [
    dict(heads=2, kv_heads=2, dim=24, vdim=40, conv=4),
    dict(heads=4, kv_heads=2, dim=64, vdim=32, conv=3),
    dict(heads=2, kv_heads=1, dim=128, vdim=128, conv=4),
    dict(heads=3, kv_heads=3, dim=10, vdim=7, conv=1),
    dict(heads=2, kv_heads=2, dim=64, vdim=64, conv=6),
]
DELTA_WIDTHS = [40, 64, 128, 44, 72]


def delta_mixer(spec, weights, width):
    return ChannelDelta(cuda(weights), width=width, heads=spec["heads"], kv_heads=spec["kv_heads"], dim=spec["dim"],
                        vdim=spec["vdim"], epsilon=EPS)


@BOTH
@pytest.mark.parametrize("index", range(len(DELTA)))
def test_channel_delta(dtype, index):
    spec, width = DELTA[index], DELTA_WIDTHS[index]
    weights = mixer_weights("channel_delta", spec, width, dtype, gate_rank=[5, 16, 20, 8, 3][index], seed=index)
    h = random_rows(150, width, dtype, 20 + index)
    want = oracle.channel_delta(double(weights), spec, h.double(), EPS)
    mixer = delta_mixer(spec, weights, width)
    for cuts in CUTS:
        close(run_mixer(mixer, h, cuts), want, dtype)


@BOTH
@pytest.mark.parametrize("shift", [-9.0, 1.0, 8.0])
def test_channel_delta_at_extreme_decays(dtype, shift):
    """Decays next to 1 (state of the first tokens intact at the end) and next to 0 (products of decays
    underflow inside a chunk: nothing may become inf or NaN)."""
    spec, width = DELTA[1], 64
    weights = mixer_weights("channel_delta", spec, width, dtype, seed=7)
    weights["dt_bias"] = torch.full_like(weights["dt_bias"], shift)
    weights["dt_bias"][::3] -= 6.0  # neighbouring channels at very different rates
    weights["A_log"] = torch.full_like(weights["A_log"], 1.5)
    h = random_rows(200, width, dtype, 8)
    want = oracle.channel_delta(double(weights), spec, h.double(), EPS)
    mixer = delta_mixer(spec, weights, width)
    for cuts in ([200], [1] * 200, [100, 2, 98]):
        close(run_mixer(mixer, h, cuts), want, dtype, 1.5)


def test_delta_write_is_read_by_its_own_token_and_erased_by_the_next():
    """One direction written, read in the same step, overwritten later: beta near 1, no decay."""
    spec = dict(heads=1, kv_heads=1, dim=16, vdim=16, conv=1)
    weights = mixer_weights("channel_delta", spec, 32, torch.float32, seed=3)
    weights["dt_bias"] = torch.full_like(weights["dt_bias"], -30.0)
    weights["a2"] = torch.zeros_like(weights["a2"])
    h = random_rows(70, 32, torch.float32, 4)
    h[69] = h[0]  # the same key as the first token, long after it
    mixer = delta_mixer(spec, weights, 32)
    want = oracle.channel_delta(double(weights), spec, h.double(), EPS)
    for cuts in ([70], [69, 1], [35, 35]):
        close(run_mixer(mixer, h, cuts), want, torch.float32)


@pytest.mark.parametrize("kind", ["retention", "delta"])
@pytest.mark.parametrize("dim,vdim", [(64, 64), (40, 24), (128, 128), (100, 50)])
def test_chunked_recurrence_equals_the_scan(kind, dim, vdim):
    """The tensor-core form against the token-by-token fp32 scan on the same operands: split operands keep
    far more than bf16 would. Several sequences of one step, one of them continued, strong and weak decays."""
    heads, kv_heads = 4, 4 if kind == "retention" else 2
    counts, bases = [1, 63, 64, 65, 200], [0, 5, 0, 64, 17]
    batch = batch_of([(4 - i, bases[i], counts[i]) for i in range(5)])
    g = torch.Generator(device="cuda").manual_seed(dim)
    rand = lambda *shape: torch.randn(*shape, generator=g, device="cuda")
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q, k = unit(rand(batch.rows, kv_heads, dim)), unit(rand(batch.rows, kv_heads, dim))
    v = rand(batch.rows, heads, vdim)
    if kind == "retention":
        beta, decay = None, torch.tensor([0.05, 0.9, 0.999, 1.0], device="cuda")
    else:
        beta = torch.sigmoid(rand(batch.rows, heads))
        decay = -torch.exp(3 * rand(batch.rows, heads, dim) - 3)
        decay[::7, 1] = -200.0  # a token that forgets everything
    start = rand(5, heads, dim, (vdim + 3) // 4 * 4)
    start[..., vdim:] = 0
    states = [start.clone(), start.clone()]
    want = hk.recurrence_scan(q, k, v, beta, decay, states[0], batch)
    got = hk.recurrence_chunked(q, k, v, beta, decay, states[1], batch)
    assert bool(torch.isfinite(got).all())
    for a, b in ((got, want), (states[1], states[0])):
        assert float((a - b).abs().max()) <= 2e-4 * float(b.abs().max())


# ------------------------------------------------------------------- latent attention ----
LATENT = [
    dict(heads=3, dim=24, vdim=40, q_rank=28, kv_rank=36, scale=0.2),
    dict(heads=5, dim=64, vdim=48, q_rank=64, kv_rank=80, scale=0.125),
    dict(heads=2, dim=128, vdim=128, q_rank=72, kv_rank=128, scale=0.09),
    dict(heads=20, dim=16, vdim=16, q_rank=20, kv_rank=20, scale=0.3),
    dict(heads=2, dim=144, vdim=20, q_rank=32, kv_rank=272, scale=0.08),
]
LATENT_WIDTHS = [40, 64, 36, 128, 72]


def latent_mixer(spec, weights, width, kv_from=None):
    return LatentAttention(cuda(weights), width=width, heads=spec["heads"], dim=spec["dim"], vdim=spec["vdim"],
                           q_rank=spec["q_rank"], kv_rank=spec["kv_rank"], scale=spec["scale"], epsilon=EPS,
                           kv_from=kv_from)


@BOTH
@pytest.mark.parametrize("index", range(len(LATENT)))
def test_latent_attention(dtype, index):
    spec, width = LATENT[index], LATENT_WIDTHS[index]
    weights = mixer_weights("latent_attention", spec, width, dtype, seed=index)
    h = random_rows(150, width, dtype, 30 + index)
    w = double(weights)
    want = oracle.latent_attention(w, spec, h.double(), oracle.latent_rows(w, h.double(), EPS), EPS)
    mixer = latent_mixer(spec, weights, width)
    for cuts in CUTS:
        close(run_mixer(mixer, h, cuts), want, dtype)


@BOTH
@pytest.mark.parametrize("sink", [-40.0, 3.0, 12.0])
def test_sink_takes_its_share_of_the_denominator(dtype, sink):
    spec, width = LATENT[1], 64
    weights = mixer_weights("latent_attention", spec, width, dtype, seed=5)
    weights["sink"] = torch.full_like(weights["sink"], sink)
    h = random_rows(140, width, dtype, 6)
    w = double(weights)
    latent = oracle.latent_rows(w, h.double(), EPS)
    want = oracle.latent_attention(w, spec, h.double(), latent, EPS)
    mixer = latent_mixer(spec, weights, width)
    for cuts in ([140], [1] * 140, [70, 70]):
        got = run_mixer(mixer, h, cuts)
        for rows in (slice(0, 2), slice(2, 140)):  # with one key the sink matters most
            close(got[rows], want[rows], dtype)


@pytest.mark.parametrize("dtype,rank,heads", [(torch.float32, 48, 3), (torch.bfloat16, 64, 3),
                                              (torch.bfloat16, 512, 16), (torch.bfloat16, 80, 70),
                                              (torch.bfloat16, 256, 28), (torch.bfloat16, 512, 40)],
                         ids=["fp32", "bf16", "rank512", "70heads", "rank256", "rank512-40heads"])
@pytest.mark.parametrize("tokens", [1, 3])
@pytest.mark.parametrize("path", ["tcgen05", "mma.sync"])
def test_one_key_that_stands_out(dtype, rank, heads, tokens, path, monkeypatch):
    """Queries that match one far key: it must be found wherever it lies, and must not be seen one
    position beyond the row. Both split-KV kernels; rows behind the last key hold anything finite."""
    monkeypatch.setenv("B200_LATENT_PATH", path)
    g = torch.Generator().manual_seed(rank + heads)
    capacity, last = 700, 650  # the rows stand at last .. last + tokens - 1
    cache = (0.05 * torch.randn(2, capacity, rank, generator=g)).to(dtype).cuda()
    q = torch.randn(tokens, heads, rank, generator=g).to(dtype)
    key = torch.sign(torch.randn(rank, generator=g))
    q += 2 * key
    batch = batch_of([(1, last, tokens)])
    for position in (0, 1, 31, 32, 63, 64, 127, 128, 255, 256, 511, 512, last - 1, last, last + 1, last + 2, last + 3):
        marked = cache.clone()
        marked[1, position] = 2 * key.to(dtype).cuda()
        out = hk.latent_attention(q.cuda(), marked, None, batch, scale=0.5)
        rows = marked[1].double().cpu()
        for t in range(tokens):
            scores = torch.einsum("hr,kr->hk", q[t].double(), rows[:last + t + 1]) * 0.5
            want = torch.softmax(scores, -1) @ rows[:last + t + 1]
            close(out[t], want, dtype)
            seen = float((out[t].double().cpu() - rows[position]).abs().max()) < 0.2
            assert seen == (position <= last + t)
    kernels.runtime().check_status()


def test_latent_attention_over_ragged_batches_and_growing_scores():
    """Contexts of one key to several tiles, an idle row, and scores that grow along the context, so that the
    running reference has to move again and again."""
    g = torch.Generator().manual_seed(0)
    heads, rank, capacity = 20, 192, 1100
    lengths = [1, 2, 127, 128, 129, 700, 1099, 5]
    cache = torch.randn(9, capacity, rank, generator=g).to(torch.bfloat16)
    direction = torch.randn(rank, generator=g)
    direction /= direction.norm()
    ramp = torch.linspace(0, 60, capacity)[:, None] * direction
    cache = (0.3 * cache.float() + ramp).to(torch.bfloat16)
    q = (torch.randn(8, heads, rank, generator=g) + 4 * direction).to(torch.bfloat16)
    batch = batch_of([(slot, n - 1, 1) for slot, n in enumerate(lengths)])
    batch.slots[7] = -1
    sink = torch.randn(heads, generator=g).to(torch.bfloat16)
    out = hk.latent_attention(q.cuda(), cache.cuda(), sink.cuda(), batch, scale=0.7)
    kernels.runtime().check_status()
    assert torch.all(out[7] == 0)
    for i, n in enumerate(lengths[:7]):
        rows = cache[i, :n].double()
        scores = torch.cat([torch.einsum("hr,kr->hk", q[i].double(), rows) * 0.7, sink.double()[:, None]], -1)
        close(out[i], torch.softmax(scores, -1)[:, :-1] @ rows, torch.bfloat16)


@pytest.mark.parametrize("size", [64, 128])
@pytest.mark.parametrize("context", [0, 1, 63, 64, 127, 128, 129, 300])
def test_portion_attention_on_the_prefill_kernel(size, context):
    """Rows behind a context of any length: the diagonal crosses two key tiles. One key stands out, at
    tile borders, at a row's own position and just beyond it; the sink takes its share."""
    heads, tokens = 3, 150
    g = torch.Generator().manual_seed(context + size)
    q = torch.randn(1, heads, tokens, size, generator=g).to(torch.bfloat16)
    k = (0.1 * torch.randn(1, heads, context + tokens, size, generator=g)).to(torch.bfloat16)
    v = torch.randn(1, heads, context + tokens, size, generator=g).to(torch.bfloat16)
    sink = torch.tensor([-20.0, 0.5, 4.0]).to(torch.bfloat16)
    mark = torch.sign(torch.randn(size, generator=g)).to(torch.bfloat16)
    q += mark
    for position in {0, 127, 128, context, context + 1, context + 40, context + 149}:
        if position >= context + tokens:
            continue
        marked = k.clone()
        marked[0, :, position] = mark
        for terms in (sink, None):
            out = torch.empty(1, tokens, heads, size, dtype=torch.bfloat16, device="cuda")
            hk.context_attention(q.cuda(), marked.cuda(), v.cuda(), None if terms is None else terms.cuda(), out,
                                 context=context, scale=size ** -0.5)
            kernels.runtime().check_status()
            scores = torch.einsum("bhtd,bhkd->bhtk", q.double(), marked.double()) * size ** -0.5
            seen = torch.arange(context + tokens)[None, :] <= context + torch.arange(tokens)[:, None]
            scores.masked_fill_(~seen, -torch.inf)
            extra = torch.full((1, heads, tokens, 1), -torch.inf, dtype=torch.float64)
            if terms is not None:
                extra = terms.double()[None, :, None, None].expand_as(extra)
            weights = torch.softmax(torch.cat([scores, extra], -1), -1)[..., :-1]
            want = torch.einsum("bhtk,bhkd->bthd", weights, v.double())
            close(out[0], want[0], torch.bfloat16)


@BOTH
def test_layers_that_share_latents(dtype):
    """A layer that reads another layer's latents: its own W_uk, W_uv and queries on the other's rows."""
    spec, width = LATENT[1], 64
    config = bazirax.BaziraxConfig(vocab_size=32, hidden_size=width, norm_eps=EPS, layers=(
        bazirax.LayerSpec("latent_attention", spec, 48),
        bazirax.LayerSpec("retention", RETENTION[1], None),
        bazirax.LayerSpec("latent_attention", dict(spec, heads=3, dim=32, q_rank=24, kv_from=0), 40)))
    check_model(config, dtype, [90], [[90], [1] * 30 + [60], [50, 2, 38]])


# ------------------------------------------------------------------------ whole model ----
def small_config(variant=0):
    layers = (
        bazirax.LayerSpec("channel_delta", DELTA[1], 72),
        bazirax.LayerSpec("latent_attention", LATENT[1], 56),
        bazirax.LayerSpec("retention", RETENTION[1], 64),
        bazirax.LayerSpec("latent_attention", dict(LATENT[0], kv_rank=80, kv_from=1), None),
        bazirax.LayerSpec("channel_delta", DELTA[0], 20),
        bazirax.LayerSpec("retention", RETENTION[0], 44),
    )
    if variant == 1:
        layers = (layers[2], layers[0], layers[1])
    return bazirax.BaziraxConfig(vocab_size=[101, 96][variant], hidden_size=[60, 64][variant], norm_eps=[1e-5, 1e-3][variant],
                                 layers=layers)


def model(config, dtype, *, batch=3, capacity=256, seed=0):
    weights = bazirax.make_weights(config, seed=seed, dtype=dtype, gate_rank=12)
    return HybridEngine(config, cuda(weights), batch=batch, capacity=capacity), weights


def check_model(config, dtype, lengths, cut_lists):
    engine, weights = model(config, dtype)
    for seed, length in enumerate(lengths):
        tokens = tokens_of(config, length, seed)
        want = oracle.forward(config.to_dict(), weights, tokens)
        for cuts in cut_lists:
            got = run_cut(engine, tokens, cuts)
            close(got, want, dtype, MODEL_TOLERANCE[dtype])
            typical = (got.double().cpu() - want).pow(2).mean(-1).sqrt().median() / want.pow(2).mean(-1).sqrt().max()
            assert float(typical) <= TOLERANCE[dtype]


@BOTH
@pytest.mark.parametrize("variant", [0, 1])
def test_model_in_portions(dtype, variant):
    """Whole, token by token, two tokens at a time, odd cuts: one logit row per position."""
    check_model(small_config(variant), dtype, [140],
                [[140], [1] * 140, [2] * 70, [3, 64, 2, 66, 5], [130, 1, 1, 1, 1, 1, 5]])


@BOTH
def test_residual_stream_after_every_layer(dtype):
    config = small_config()
    engine, weights = model(config, dtype)
    tokens = tokens_of(config, 40, 1)
    want, got = [], []
    oracle.forward(config.to_dict(), weights, tokens, streams=want)
    slot = engine.open()
    engine.forward([(slot, tokens)], streams=got)
    assert len(got) == len(want) == config.num_layers
    for a, b in zip(got, want):
        assert a.dtype == torch.float32
        close(a, b, dtype, MODEL_TOLERANCE[dtype])


@BOTH
def test_first_tokens(dtype):
    """Sequences of one, two and three tokens: empty convolution history, one key, an empty state."""
    config = small_config()
    engine, weights = model(config, dtype)
    for length in (1, 2, 3):
        tokens = tokens_of(config, length, length)
        want = oracle.forward(config.to_dict(), weights, tokens)
        close(run_cut(engine, tokens, [length]), want, dtype, MODEL_TOLERANCE[dtype])
        close(run_cut(engine, tokens, [1] * length), want, dtype, MODEL_TOLERANCE[dtype])


def test_equal_prompts_in_one_step_equal_each_alone():
    """Whole prompts of one length take one attention launch over the step's own latents."""
    config = small_config()
    engine, weights = model(config, torch.bfloat16)
    prompts = [tokens_of(config, 140, s) for s in range(3)]
    slots = [engine.open() for _ in prompts]
    got = engine.forward(list(zip(slots, prompts)), [list(range(140))] * 3)
    for i, prompt in enumerate(prompts):
        close(got[140 * i:140 * (i + 1)], oracle.forward(config.to_dict(), weights, prompt), torch.bfloat16,
              MODEL_TOLERANCE[torch.bfloat16])


@BOTH
def test_unequal_batches_equal_each_alone(dtype):
    """Whole prompts, portions and decoded tokens of several sequences in one step."""
    config = small_config()
    engine, weights = model(config, dtype, batch=4)
    sequences = [tokens_of(config, n, 50 + n) for n in (90, 17, 3, 130)]
    want = [oracle.forward(config.to_dict(), weights, s) for s in sequences]
    slots = [engine.open() for _ in sequences]
    plan = [[(0, 40), (1, 10), (3, 1)], [(3, 70), (0, 1), (2, 2)], [(1, 1), (2, 1), (3, 1), (0, 1)],
            [(0, 48), (1, 6), (3, 58)]]
    at = [0] * 4
    for step in plan:
        entries = [(slots[i], sequences[i][at[i]:at[i] + n]) for i, n in step]
        got = engine.forward(entries, [list(range(n)) for _, n in step])
        first = 0
        for i, n in step:
            close(got[first:first + n], want[i][at[i]:at[i] + n], dtype, MODEL_TOLERANCE[dtype])
            first += n
            at[i] += n
    assert at == [90, 17, 3, 130]
    engine.state.check()


def test_slots_are_used_again_and_do_not_mix():
    """A slot whose former sequence was longer gives what a fresh engine gives, bit for bit."""
    config = small_config()
    engine, _ = model(config, torch.bfloat16, batch=2)
    long, short = tokens_of(config, 200, 1), tokens_of(config, 33, 2)
    fresh = run_cut(engine, short, [20, 13])
    for _ in range(3):
        run_cut(engine, long, [200])
        assert torch.equal(run_cut(engine, short, [20, 13]), fresh)
    a, b = engine.open(), engine.open()
    with pytest.raises(ExecutionError):
        engine.open()
    engine.forward([(a, long[:50]), (b, short[:5])])
    engine.close(a)
    c = engine.open()
    assert c == a
    together = engine.forward([(c, short)], [list(range(33))])
    close(together, fresh.double().cpu(), torch.bfloat16, MODEL_TOLERANCE[torch.bfloat16])
    assert engine.state.slots_in_use() == 2


def test_step_arguments_are_checked():
    config = small_config()
    engine, _ = model(config, torch.float32, capacity=16)
    slot = engine.open()
    with pytest.raises(ValueError):
        engine.forward([(slot, [])])
    with pytest.raises(ValueError):
        engine.forward([(slot, [1]), (slot, [2])])
    with pytest.raises(ValueError):
        engine.forward([(slot, [1, 2])], [[2]])
    with pytest.raises(ExecutionError):
        engine.forward([(slot, [1] * 17)])
    engine.forward([(slot, [1] * 16)])
    with pytest.raises(ExecutionError):
        engine.decode_rows([slot], [1])


@BOTH
def test_long_decoding(dtype):
    """Hundreds of decoded tokens from captured steps against the whole sequence at once."""
    config = small_config(1)
    engine, weights = model(config, dtype, batch=2, capacity=512)
    tokens = tokens_of(config, 400, 9)
    want = oracle.forward(config.to_dict(), weights, tokens)
    slot = engine.open()
    engine.forward([(slot, tokens[:10])])
    for place in range(10, 400):
        engine.decode_rows([slot], [tokens[place]])
        if place % 39 == 0 or place == 399:
            close(engine.logits, want[place:place + 1], dtype, MODEL_TOLERANCE[dtype])
    engine.state.check()


@BOTH
def test_scheduler_generates_what_the_oracle_generates(dtype):
    """Greedy generation of unequal requests, more of them than slots, prompts in portions; teacher-forced
    margin where a bf16 near-tie falls the other way."""
    config = small_config(1)
    engine, weights = model(config, dtype, batch=3, capacity=128)
    scheduler = RequestScheduler(engine, max_portion=16)
    requests = [scheduler.submit(tokens_of(config, n, 70 + n), 5) for n in (40, 3, 17, 1, 29)]
    scheduler.run()
    for request in requests:
        assert request.finished and len(request.output) == 5
        logits = oracle.forward(config.to_dict(), weights, request.prompt + request.output)
        scale = float(logits.abs().max())
        for i, token in enumerate(request.output):
            row = logits[len(request.prompt) - 1 + i]
            assert float(row.max() - row[token]) <= (1e-4 if dtype == torch.float32 else 6e-2) * scale
    assert engine.state.slots_in_use() == 0


def test_generate_equals_the_scheduler_and_the_uncaptured_step():
    config = small_config(1)
    engine, _ = model(config, torch.bfloat16, batch=3, capacity=128)
    prompts = torch.tensor([tokens_of(config, 24, s) for s in range(3)])
    captured = engine.generate(prompts, 6)
    eager = engine.generate(prompts, 6, use_graph=False)
    other, _ = model(config, torch.bfloat16, batch=3, capacity=128)
    uncaptured = other.generate(prompts, 6, use_graph=False)
    assert torch.equal(captured, eager) and torch.equal(captured, uncaptured)
    step = other.step(captured[:, -1].cpu())
    assert step.shape == (3,)
    scheduled, _ = model(config, torch.bfloat16, batch=3, capacity=128)
    scheduler = RequestScheduler(scheduled)
    requests = [scheduler.submit(p, 7) for p in prompts.tolist()]
    scheduler.run()
    assert [r.output for r in requests] == captured.tolist()


def test_idle_rows_leave_no_trace():
    """A decode batch rounded up with idle rows changes nothing of the slots that sit out."""
    config = small_config(1)
    engine, _ = model(config, torch.bfloat16, batch=4, capacity=64)
    slots = [engine.open() for _ in range(4)]
    for i, slot in enumerate(slots):
        engine.forward([(slot, tokens_of(config, 5 + i, i))])
    before = [{k: v[slots[3]].clone() for k, v in layer.items()} for layer in engine.state.layers]
    engine.decode_rows(slots[:3], [1, 2, 3])  # four rows, one idle
    for layer, saved in zip(engine.state.layers, before):
        for name, tensor in layer.items():
            assert torch.equal(tensor[slots[3]], saved[name])
    assert engine.state.lengths.tolist() == [6, 7, 8, 8]


# ---------------------------------------------------------------- files and command line ----
def stored_model(folder, config, seed=0):
    weights = bazirax.make_weights(config, seed=seed, dtype=torch.bfloat16, gate_rank=12)
    (folder / "config.json").write_text(json.dumps(config.to_dict()))
    save_safetensors(weights, folder / "model.safetensors")
    return weights


@BOTH
def test_trace_replay(dtype, tmp_path):
    """A stored model loaded through the registry and driven step by step: portions, a step without wanted
    places, a second sequence in the slot of the first."""
    config = small_config(1)
    weights = stored_model(tmp_path, config)
    first, second = tokens_of(config, 60, 1), tokens_of(config, 25, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": first[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": first[50:58], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": first[58:], "want": [1, 0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": second, "want": [24]}], "end": ["b"]}]
    output = io.StringIO()
    engine = load_model(tmp_path, dtype=dtype, batch=1, capacity=64)
    replay(engine, [json.dumps(step) for step in steps], tmp_path, output)
    assert output.getvalue().split("\n")[:-1] == [f"done {n}" for n in range(4)]
    assert not (tmp_path / "1.f32").exists() and engine.state.slots_in_use() == 0
    a, b = (oracle.forward(config.to_dict(), weights, t) for t in (first, second))
    for step, want in ((0, a[[0, 49]]), (2, a[[59, 58]]), (3, b[[24]])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(want), config.vocab_size)
        close(torch.from_numpy(got), want, dtype, MODEL_TOLERANCE[dtype])


def test_command_line_generates_from_a_stored_model(tmp_path, capsys):
    config = small_config(1)
    stored_model(tmp_path, config, seed=3)
    prompts = [tokens_of(config, n, n) for n in (5, 30, 11)]
    arguments = [x for p in prompts for x in ("--prompt", ",".join(map(str, p)))]
    assert main(["generate", "--model", str(tmp_path), "--new-tokens", "4", "--max-batch", "2", "--max-portion", "8",
                 *arguments]) == 0
    lines = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    assert [line["prompt"] for line in lines] == prompts
    engine, _ = model(config, torch.bfloat16, batch=2, capacity=34, seed=3)
    scheduler = RequestScheduler(engine, max_portion=8)
    requests = [scheduler.submit(p, 4) for p in prompts]
    scheduler.run()
    assert [line["output"] for line in lines] == [r.output for r in requests]
