"""The Lozanex design on the GPU against the plain implementation of oracle/hybrid_model.py: attention within
chunks, the delta rule with one decay per head and the mixture of experts alone, then whole models: portions
of any size, token-by-token decoding, unequal batches, slots that are used again, long decoding and greedy
generation through the scheduler."""

import io
import json

import numpy as np
import pytest
import torch

from hybrid_helpers import (BOTH, CUTS, EPS, MODEL_TOLERANCE, TOLERANCE, batch_of, close, cuda, double, random_rows,
                            run_cut, run_mixer, summed, tokens_of)
from llm_compiler_b200 import hybrid_kernels as hk
from llm_compiler_b200 import kernels, lozanex
from llm_compiler_b200.cli import main
from llm_compiler_b200.hybrid_engine import HybridEngine
from llm_compiler_b200.mixers import Attention, ExpertMlp, HeadDelta
from llm_compiler_b200.registry import load_model
from llm_compiler_b200.safetensors_io import save_safetensors
from llm_compiler_b200.scheduler import RequestScheduler
from llm_compiler_b200.trace import replay
from oracle import hybrid_model as oracle

pytestmark = pytest.mark.gpu


def layer_weights(kind, spec, width, dtype, *, mlp=None, seed=0):
    config = lozanex.LozanexConfig(vocab_size=8, hidden_size=width, norm_eps=EPS,
                                   layers=(lozanex.LayerSpec(kind, spec, mlp),))
    part = "l0.mix." if mlp is None else "l0.mlp."
    return {name[len(part):]: w for name, w in lozanex.make_weights(config, seed=seed, dtype=dtype).items()
            if name.startswith(part)}


# ---------------------------------------------------------------------- norms, embedding ----
@BOTH
@pytest.mark.parametrize("width", [48, 54, 1000, 2600])
@pytest.mark.parametrize("rows", [3, 400])
def test_residual_norm_adds_a_bias_and_scattered_rows(dtype, width, rows):
    g = torch.Generator().manual_seed(width)
    wide = hk.pad8(width)
    x = torch.randn(rows, width, generator=g)
    y, pool = torch.randn(rows, wide, generator=g).to(dtype), torch.randn(50, wide, generator=g).to(dtype)
    bias, post, after = (torch.randn(3, width, generator=g)).to(dtype)
    places = torch.randint(0, 50, (rows, 3), generator=g, dtype=torch.int32)
    picked = pool.double()[places.long()].sum(1)[:, :width]
    for parts, total in ((hk.Summands(y.cuda(), bias.cuda(), pool.cuda(), places.cuda()),
                          y.double()[:, :width] + bias.double() + picked),
                         (hk.Summands(None, None, pool.cuda(), places.cuda()), picked),
                         (hk.Summands(torch.stack([y.float(), y.float()]).cuda(), bias.cuda()),
                          2 * y.double()[:, :width] + bias.double())):
        want = x.double() + oracle.rms_norm(total, post.double(), EPS)
        residual = x.cuda()
        h = hk.residual_norm(residual, parts, post.cuda(), None, epsilon=EPS, weight_offset=0.0, dtype=dtype, narrow=True)
        assert float((residual.double().cpu() - want).abs().max()) < 2e-5
        assert torch.equal(h[:, :width], residual.to(dtype)) and torch.all(h[:, width:] == 0)
        residual = x.cuda()
        h = hk.residual_norm(residual, parts, post.cuda(), after.cuda(), epsilon=EPS, weight_offset=0.0, dtype=dtype)
        close(h[:, :width], oracle.rms_norm(want, after.double(), EPS), dtype)


@BOTH
@pytest.mark.parametrize("width", [36, 50, 1100])
def test_embedding_with_a_norm(dtype, width):
    table = torch.randn(11, width, generator=torch.Generator().manual_seed(0)).to(dtype)
    weight = (1 + 0.2 * torch.randn(width, generator=torch.Generator().manual_seed(1))).to(dtype)
    ids = torch.tensor([3, 0, 10, 3])
    x, h = hk.embedding_residual(table.cuda(), ids.cuda(), weight.cuda(), epsilon=EPS, narrow=True)
    want = oracle.rms_norm(table.double()[ids], weight.double(), EPS)
    assert float((x.double().cpu() - want).abs().max()) < 1e-5
    assert torch.equal(h[:, :width], x.to(dtype)) and torch.all(h[:, width:] == 0)
    x = hk.embedding_residual(table.cuda(), torch.tensor([11, 2]).cuda(), weight.cuda(), epsilon=EPS)
    with pytest.raises(kernels.KernelStatusError, match="token id"):
        kernels.runtime().check_status()
    assert torch.all(x[0] == 0)


# ------------------------------------------------------------------------- delta rule ----
DELTA = [
    dict(heads=2, kv_heads=2, dim=24, vdim=40, conv=4),
    dict(heads=6, kv_heads=2, dim=64, vdim=64, conv=3),
    dict(heads=2, kv_heads=1, dim=128, vdim=128, conv=4),
    dict(heads=3, kv_heads=3, dim=10, vdim=7, conv=1),
    dict(heads=4, kv_heads=2, dim=128, vdim=64, conv=2),
    dict(heads=1, kv_heads=1, dim=1, vdim=5, conv=6),
    dict(heads=2, kv_heads=2, dim=144, vdim=32, conv=4),
]
DELTA_WIDTHS = [40, 64, 128, 44, 72, 30, 56]


def delta_mixer(spec, weights, width):
    return HeadDelta(cuda(weights), width=width, heads=spec["heads"], kv_heads=spec["kv_heads"], dim=spec["dim"],
                     vdim=spec["vdim"], epsilon=EPS)


@BOTH
@pytest.mark.parametrize("index", range(len(DELTA)))
def test_head_delta(dtype, index):
    spec, width = DELTA[index], DELTA_WIDTHS[index]
    weights = layer_weights("delta", spec, width, dtype, seed=index)
    h = random_rows(150, width, dtype, 20 + index)
    want = oracle.head_delta(double(weights), spec, h.double(), EPS)
    mixer = delta_mixer(spec, weights, width)
    for cuts in CUTS:
        close(run_mixer(mixer, h, cuts), want, dtype, 1.5)


@BOTH
@pytest.mark.parametrize("shift", [-9.0, 1.0, 8.0])
def test_head_delta_at_extreme_decays(dtype, shift):
    """Decays next to 1 (what the first tokens wrote is intact at the end) and next to 0 (products of decays
    underflow inside a chunk)."""
    spec, width = DELTA[1], 64
    weights = layer_weights("delta", spec, width, dtype, seed=7)
    weights["dt_bias"] = torch.full_like(weights["dt_bias"], shift)
    weights["dt_bias"][::3] -= 6.0  # neighbouring heads at very different rates
    weights["A_log"] = torch.full_like(weights["A_log"], 1.5)
    h = random_rows(200, width, dtype, 8)
    want = oracle.head_delta(double(weights), spec, h.double(), EPS)
    mixer = delta_mixer(spec, weights, width)
    for cuts in ([200], [1] * 200, [100, 2, 98]):
        close(run_mixer(mixer, h, cuts), want, dtype, 1.5)


@pytest.mark.parametrize("dim,vdim", [(64, 64), (40, 24), (128, 128), (100, 50), (1, 20)])
def test_chunked_head_delta_equals_the_scan(dim, vdim):
    """The tensor-core form against the token-by-token fp32 scan on the same operands: several sequences of one
    step, some continued, decays from 1 to nothing."""
    heads, kv_heads = 4, 2
    counts, bases = [1, 63, 64, 65, 200], [0, 5, 0, 64, 17]
    batch = batch_of([(4 - i, bases[i], counts[i]) for i in range(5)])
    g = torch.Generator(device="cuda").manual_seed(dim)
    rand = lambda *shape: torch.randn(*shape, generator=g, device="cuda")
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q, k = unit(rand(batch.rows, kv_heads, dim)), unit(rand(batch.rows, kv_heads, dim))
    v = rand(batch.rows, heads, vdim)
    beta = torch.sigmoid(rand(batch.rows, heads))
    decay = -torch.exp(3 * rand(batch.rows, heads, 1) - 3)
    decay[::7, 1] = -200.0  # a token that forgets everything
    decay[:, 2] = 0.0
    start = rand(5, heads, dim, (vdim + 3) // 4 * 4)
    start[..., vdim:] = 0
    states = [start.clone(), start.clone()]
    want = hk.recurrence_scan(q, k, v, beta, decay, states[0], batch)
    got = hk.recurrence_chunked(q, k, v, beta, decay, states[1], batch)
    assert bool(torch.isfinite(got).all())
    for a, b in ((got, want), (states[1], states[0])):
        assert float((a - b).abs().max()) <= 2e-4 * float(b.abs().max())


def test_a_decay_per_head_equals_equal_decays_per_channel():
    heads, dim, vdim = 3, 64, 48
    batch = batch_of([(1, 9, 130), (0, 0, 70)])
    g = torch.Generator(device="cuda").manual_seed(1)
    rand = lambda *shape: torch.randn(*shape, generator=g, device="cuda")
    q, k = (x / x.norm(dim=-1, keepdim=True) for x in (rand(200, heads, dim), rand(200, heads, dim)))
    v, beta, decay = rand(200, heads, vdim), torch.sigmoid(rand(200, heads)), -torch.exp(rand(200, heads, 1) - 2)
    start = rand(2, heads, dim, vdim)
    for form in (hk.recurrence_scan, hk.recurrence_chunked):
        one, per_channel = start.clone(), start.clone()
        a = form(q, k, v, beta, decay, one, batch)
        b = form(q, k, v, beta, decay.expand(-1, -1, dim).contiguous(), per_channel, batch)
        assert float((a - b).abs().max()) < 2e-4 and float((one - per_channel).abs().max()) < 2e-4


# -------------------------------------------------------------------------- attention ----
ATTENTION = [
    dict(heads=6, kv_heads=2, dim=24, vdim=40, scale=0.3, rot=dict(base=1e4, dims=16), mask=dict(size=48)),
    dict(heads=4, kv_heads=4, dim=64, vdim=64, scale=0.125, rot=dict(base=1e6, dims=64), mask=dict(size=64)),
    dict(heads=5, kv_heads=1, dim=128, vdim=80, scale=0.07, rot=dict(base=500.0, dims=2), mask=dict(size=33)),
    dict(heads=2, kv_heads=1, dim=72, vdim=128, scale=0.2, rot=None, mask=None),
    dict(heads=20, kv_heads=1, dim=32, vdim=16, scale=0.2, rot=dict(base=1e4, dims=8), mask=dict(size=1)),
    dict(heads=2, kv_heads=2, dim=150, vdim=30, scale=0.1, rot=dict(base=1e5, dims=100), mask=dict(size=100)),
    dict(heads=3, kv_heads=3, dim=13, vdim=9, scale=0.4, rot=dict(base=1e4, dims=6), mask=dict(size=7)),
    dict(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15, rot=dict(base=1e4, dims=32), mask=dict(size=1000)),
]
ATTENTION_WIDTHS = [40, 64, 36, 128, 72, 52, 44, 96]


def attention_mixer(spec, weights, width, **more):
    dims, base = lozanex._rotation(spec)
    return Attention(cuda(weights), width=width, heads=spec["heads"], kv_heads=spec["kv_heads"], dim=spec["dim"],
                     vdim=spec["vdim"], scale=spec["scale"], rot_dims=dims, rot_base=base, epsilon=EPS,
                     chunk=None if spec["mask"] is None else spec["mask"]["size"], **more)


@BOTH
@pytest.mark.parametrize("index", range(len(ATTENTION)))
def test_attention(dtype, index):
    spec, width = ATTENTION[index], ATTENTION_WIDTHS[index]
    weights = layer_weights("attention", spec, width, dtype, seed=index)
    h = random_rows(150, width, dtype, 30 + index)
    w = double(weights)
    want = oracle.attention(w, spec, h.double(), *oracle.attention_keys(w, spec, h.double(), EPS), EPS)
    mixer = attention_mixer(spec, weights, width)
    for cuts in CUTS:
        close(run_mixer(mixer, h, cuts), want, dtype)


@BOTH
def test_norms_span_the_whole_projection(dtype):
    """A head of large queries (or keys) shrinks the others: the norm is over the projection, not per head, and
    the bias is inside it."""
    spec, width = ATTENTION[0], 40
    weights = layer_weights("attention", spec, width, dtype, seed=3)
    weights["q"][:24] *= 6.0
    weights["k"][24:48] *= 5.0
    weights["q.b"][-24:] += 2.0
    h = random_rows(60, width, dtype, 4)
    w = double(weights)
    want = oracle.attention(w, spec, h.double(), *oracle.attention_keys(w, spec, h.double(), EPS), EPS)
    for cuts in ([60], [1] * 60):
        close(run_mixer(attention_mixer(spec, weights, width), h, cuts), want, dtype)


def test_far_positions_turn_exactly():
    """A product of a query and a key at far positions depends on their distance only."""
    spec = dict(ATTENTION[1], mask=None)
    weights = layer_weights("attention", spec, 64, torch.float32, seed=2)
    mixer = attention_mixer(spec, weights, 64)
    h = random_rows(4, 64, torch.float32, 3).cuda()
    products = []
    for base in (0, 100000):
        keys, values = torch.zeros(2, 1, 100004, 4, 64, device="cuda")
        q = hk.attention_prep(kernels.b200_linear(h, mixer.w_in, mixer.bias), None, mixer.q_norm, mixer.k_norm,
                              mixer.turns, keys, values, batch_of([(0, base, 4)]), heads=4, kv_heads=4, dim=64, vdim=64,
                              row_size=64, columns=mixer.columns, epsilon=EPS)
        products.append(torch.einsum("ihd,jhd->hij", q.double(), keys[0, base:base + 4].double()))
    assert float((products[0] - products[1]).abs().max()) < 1e-5 * float(products[0].abs().max())


def marked_attention(q, keys, values, row, slot, chunk, scale):
    """Plain attention of one query row [H, D] at position `row` of a slot."""
    first = row // chunk * chunk if chunk else 0
    k, v = (t[slot, first:row + 1].double().cpu() for t in (keys, values))
    group = q.shape[0] // k.shape[1]
    k, v = k.repeat_interleave(group, 1), v.repeat_interleave(group, 1)
    weights = torch.softmax(torch.einsum("hd,khd->hk", q.double().cpu(), k) * scale, -1)
    return torch.einsum("hk,khd->hd", weights, v)


@pytest.mark.parametrize("form", ["generic-fp32", "generic", "decode", "portion"])
@pytest.mark.parametrize("chunk", [0, 97, 128, 300])
@pytest.mark.parametrize("size,heads,kv_heads", [(64, 6, 2), (128, 20, 1)])
def test_one_key_that_stands_out(form, chunk, size, heads, kv_heads):
    """Queries that match one key, which lies just inside or just outside the row's chunk, far away, at tile
    borders, or one position ahead: it must weigh in exactly when the row sees it."""
    dtype = torch.float32 if form == "generic-fp32" else torch.bfloat16
    g = torch.Generator().manual_seed(chunk + size)
    capacity, slot = 700, 2
    mark = torch.sign(torch.randn(size, generator=g))
    keys = (0.05 * torch.randn(3, capacity, kv_heads, size, generator=g)).to(dtype).cuda()
    values = torch.randn(3, capacity, kv_heads, size, generator=g).to(dtype).cuda()
    q = (0.1 * torch.randn(700, heads, size, generator=g) + mark).to(dtype).cuda()
    scale = 12.0 / size
    step = chunk or 250
    rows = sorted({0, 1, step - 1, step, step + 1, 2 * step - 1, 2 * step, 600, 640})
    if form == "portion":  # all rows between two of them in one launch
        spans = [(0, 300), (step - 3, 260), (599, 42), (600, 1), (2 * step, 2)]
    else:
        spans = [(row, 1) for row in rows]
    for first, count in spans:
        edge = first // chunk * chunk if chunk else 0
        marks = {edge - 1, edge, first - 1, first, first + 1, first + count - 1, first + count, edge + 127, edge + 128,
                 0, 5, 255, 256, step - 1, step, 2 * step - 1, 2 * step}
        for position in sorted(p for p in marks if 0 <= p < capacity):
            marked = keys.clone()
            marked[slot, position] = mark.to(dtype).cuda()
            part = q[first:first + count].contiguous()
            batch = batch_of([(slot, first, count)])
            if form == "decode":
                out = hk.slot_decode_attention(part, marked, values, batch, scale=scale, chunk=chunk)
            elif form == "portion":
                out = torch.empty_like(part)
                seen = slice(edge, first + count)
                hk.context_attention(part[None].transpose(1, 2), marked[slot:slot + 1, seen].transpose(1, 2),
                                     values[slot:slot + 1, seen].transpose(1, 2), None, out[None], context=first - edge,
                                     scale=scale, chunk=chunk)
            else:
                out = hk.slot_attention(part, marked, values, batch, scale=scale, chunk=chunk)
            checked = range(count) if count <= 3 else sorted({0, 1, count // 2, count - 1, *(
                r for r in (position - first - 1, position - first, position - first + 1,
                            step - 1 - first, step - first, 2 * step - 1 - first, 2 * step - first) if 0 <= r < count)})
            for r in checked:
                row = first + r
                close(out[r], marked_attention(part[r], marked, values, row, slot, chunk, scale), dtype)
                inside = position <= row and (not chunk or position // chunk == row // chunk)
                near = float((out[r].double().cpu() - values[slot, position].double().cpu()
                              .repeat_interleave(heads // kv_heads, 0)).abs().max()) < 0.3
                assert near == inside
    kernels.runtime().check_status()


@pytest.mark.parametrize("chunk", [0, 512, 700])
@pytest.mark.parametrize("size,heads,kv_heads", [(64, 14, 2), (128, 4, 4)])
def test_decode_attention_over_ragged_slots(chunk, size, heads, kv_heads):
    """Rows of unequal contexts in slots out of order, one idle, few rows (splits merged in a cluster) and many."""
    g = torch.Generator().manual_seed(size)
    capacity = 5000 if chunk == 0 else 1500
    lengths = [1, 2, 127, 128, 513, 1025, capacity, 700, 1400, 701]
    slots = [3, 9, 0, 7, 1, 2, 8, 4, 6, 5]
    keys = torch.randn(10, capacity, kv_heads, size, generator=g).to(torch.bfloat16).cuda()
    values = torch.randn(10, capacity, kv_heads, size, generator=g).to(torch.bfloat16).cuda()
    for count in (2, 10):
        picked = list(zip(slots, lengths))[-count:]
        batch = batch_of([(slot, n - 1, 1) for slot, n in picked])
        batch.slots[0] = -1
        q = torch.randn(count, heads, size, generator=g).to(torch.bfloat16).cuda()
        out = hk.slot_decode_attention(q, keys, values, batch, scale=size ** -0.5, chunk=chunk)
        kernels.runtime().check_status()
        assert torch.all(out[0] == 0)
        for i, (slot, n) in enumerate(picked[1:], 1):
            close(out[i], marked_attention(q[i], keys, values, n - 1, slot, chunk, size ** -0.5), torch.bfloat16)


@BOTH
def test_layers_that_share_keys_and_values(dtype):
    """A layer that reads another layer's keys and values with queries, a chunk, a scale and heads of its own."""
    spec, width = ATTENTION[0], 64
    config = lozanex.LozanexConfig(vocab_size=32, hidden_size=width, norm_eps=EPS, layers=(
        lozanex.LayerSpec("attention", spec, None),
        lozanex.LayerSpec("delta", DELTA[1], None),
        lozanex.LayerSpec("attention", dict(spec, heads=4, mask=dict(size=29), scale=0.5, kv_from=0), None),
        lozanex.LayerSpec("attention", dict(spec, mask=None, kv_from=0), None)))
    check_model(config, dtype, [90], [[90], [1] * 30 + [60], [50, 2, 38]])


# ---------------------------------------------------------------------------- experts ----
EXPERTS = [
    dict(kind="moe", expert=dict(ff=40), router=dict(experts=6, top=2), shared=dict(ff=56)),
    dict(kind="moe", expert=dict(ff=136), router=dict(experts=40, top=4), shared=dict(ff=24)),
    dict(kind="moe", expert=dict(ff=20), router=dict(experts=3, top=3), shared=None),
    dict(kind="moe", expert=dict(ff=64), router=dict(experts=1, top=1), shared=dict(ff=9)),
    dict(kind="moe", expert=dict(ff=9), router=dict(experts=130, top=1), shared=dict(ff=64)),
]
EXPERT_WIDTHS = [40, 264, 36, 72, 50]


def expert_mlp(spec, weights, width):
    w = cuda(weights)
    part = lambda prefix: {name: w[f"{prefix}.{name}"] for name in ("gate", "up", "down")}
    shared = None if spec["shared"] is None else part("shared")
    return ExpertMlp(w["router"], [part(f"e{e}") for e in range(spec["router"]["experts"])], width=width,
                     top=spec["router"]["top"], shared=shared)


def expert_weights(index, dtype):
    mixer = dict(heads=1, kv_heads=1, dim=8, vdim=8, conv=1)
    return layer_weights("delta", mixer, EXPERT_WIDTHS[index], dtype, mlp=EXPERTS[index], seed=index)


def padded(h, width):
    piece = torch.zeros((h.shape[0], hk.pad8(width)), dtype=h.dtype, device="cuda")
    piece[:, :width] = h.cuda()
    return piece


@BOTH
@pytest.mark.parametrize("index", range(len(EXPERTS)))
def test_mixture_of_experts(dtype, index):
    """Decode sizes (one launch for the choice, the shared expert as slices) and prompts, called one after the
    other: the counters are zero again."""
    spec, width = EXPERTS[index], EXPERT_WIDTHS[index]
    weights = expert_weights(index, dtype)
    mlp = expert_mlp(spec, weights, width)
    tiles = set()
    for rows in (1, 20, 64, 65, 128, 129, 700):
        h = random_rows(rows, width, dtype, rows)
        got = summed(mlp(padded(h, width)))[:, :width]
        tiles.add(mlp.tile_of(rows))
        close(got, oracle.expert_mlp(double(weights), spec, h.double()), dtype)
        assert torch.all(mlp.counters == 0)
    kernels.runtime().check_status()
    assert len(tiles) >= 2


@BOTH
def test_every_token_to_one_expert_and_a_score_that_matters(dtype):
    """All rows choose the same experts (several full tiles of one, none of the others), and a score near 0
    against one near 1: it scales the input of a nonlinear map, not its output."""
    spec, width = EXPERTS[0], 40
    weights = expert_weights(0, dtype)
    weights["router"] = torch.zeros_like(weights["router"])
    weights["router"][4, 0], weights["router"][1, 0] = 3.0, -1.5
    weights["router"][(0, 2, 3, 5), 0] = -40.0
    h = random_rows(300, width, dtype, 1)
    h[:, 0] = torch.linspace(0.1, 2.0, 300).to(dtype)
    scores, chosen = oracle.route(weights["router"].double(), h.double(), 2)
    assert set(map(tuple, chosen.tolist())) == {(4, 1)} and float(scores[-1, 1]) < 0.1 < 0.9 < float(scores[-1, 0])
    mlp = expert_mlp(spec, weights, width)
    close(summed(mlp(padded(h, width)))[:, :width], oracle.expert_mlp(double(weights), spec, h.double()), dtype)


@pytest.mark.parametrize("tile", [16, 32, 64, 128, 256])
@pytest.mark.parametrize("n,k", [(400, 136), (48, 24), (256, 512)])
def test_grouped_linear_tiles(tile, n, k):
    """Every tile size against plain products: experts without rows, with one, with a tile
    exactly, with more, and two that take every row."""
    g = torch.Generator().manual_seed(tile + n)
    held = [0, 1, tile, tile + 1, 0, 3 * tile - 1, 5]
    chosen = torch.cat([torch.full((c,), e, dtype=torch.int32) for e, c in enumerate(held)])
    chosen = chosen[torch.randperm(len(chosen), generator=g)].long()
    rows = len(chosen)
    logits = torch.full((rows, 8), -9.0)
    logits[torch.arange(rows), chosen] = torch.randn(rows, generator=g)
    logits[:, 7] = 50.0  # (no expert: a column of padding)
    counters = torch.zeros(8, dtype=torch.int32, device="cuda")
    x = torch.randn(rows, k, generator=g).to(torch.bfloat16).cuda()
    order, ordered = hk.expert_route(logits.cuda(), x, counters, top=1, always=2, tile=tile)
    assert torch.all(counters == 0) and torch.equal(order.chosen.cpu()[:, 0].long(), chosen)
    assert torch.allclose(order.chosen_scores.cpu()[:, 0], torch.sigmoid(logits[torch.arange(rows), chosen]), atol=1e-6)
    places = order.places.long()
    assert places.shape == (rows, 3) and len(set(places.flatten().tolist())) == 3 * rows
    assert torch.equal(order.index[places], torch.arange(rows, device="cuda", dtype=torch.int32)[:, None].expand(-1, 3))
    table = order.tiles.tolist()
    used = [t for t in table if t[0] >= 0]
    assert table[len(used):] == [[-1, 0]] * (len(table) - len(used))
    assert [sum(count for e, count in used if e == expert) for expert in range(9)] == held + [rows, rows]
    w = (torch.randn(9, n, k, generator=g) * k ** -0.5).to(torch.bfloat16).cuda()
    assert torch.equal(ordered[places], x[:, None].expand(-1, 3, -1))
    unheld = torch.ones(ordered.shape[0], dtype=torch.bool, device="cuda")
    unheld[places.flatten()] = False
    ordered[unheld] = float("nan")  # rows that no tile holds hold anything
    experts = torch.stack([torch.full_like(chosen, 7), torch.full_like(chosen, 8), chosen], 1)
    products = torch.einsum("rjnk,rk->rjn", w.double().cpu()[experts], x.double().cpu())
    scores = order.scores[places].double().cpu()[:, :, None]
    assert torch.all(scores[:, :2] == 1)
    gated = oracle.silu(scores * products[..., 0::2]) * (scores * products[..., 1::2])
    for swiglu, want in ((False, products), (True, gated)):
        got = hk.grouped_linear(ordered, w, order, swiglu=swiglu)[places]
        close(got.flatten(0, 1), want.flatten(0, 1), torch.bfloat16)
    kernels.runtime().check_status()


@BOTH
@pytest.mark.parametrize("rows,experts,top,width", [(1, 5, 1, 40), (70, 99, 5, 136), (128, 3, 3, 264), (17, 300, 12, 1032)])
def test_choice_in_one_launch(dtype, rows, experts, top, width):
    """The router's products, the choice and the order against sorted logits of double precision."""
    g = torch.Generator().manual_seed(rows)
    h = torch.randn(rows, width, generator=g).to(dtype)
    router = (torch.randn(experts, width, generator=g) * width ** -0.5).to(dtype)
    counters = torch.zeros(experts + 1, dtype=torch.int32, device="cuda")
    logits = h.double() @ router.double().T
    want = torch.topk(logits, top, dim=-1)
    for always in (0, 2):
        order = hk.expert_select(h.cuda(), router.cuda(), counters, top=top, always=always, tile=16)
        assert torch.equal(order.chosen.cpu().long(), want.indices) and torch.all(counters == 0)
        assert torch.allclose(order.chosen_scores.cpu().double(), torch.sigmoid(want.values), atol=1e-6)
        places = order.places.long()
        assert len(set(places.flatten().tolist())) == rows * (top + always)
        assert torch.equal(order.index[places[:, -1]].cpu(), torch.arange(rows, dtype=torch.int32))
        own = order.tiles[places // 16].cpu()
        assert torch.equal(own[:, always:, 0].long(), want.indices)
        assert own[:, :always, 0].tolist() == [list(range(experts, experts + always))] * rows
        assert torch.all(places.cpu() % 16 < own[..., 1])
        assert torch.equal(order.scores[places[:, always:]], order.chosen_scores)


@BOTH
@pytest.mark.parametrize("rows,tile", [(1, 16), (16, 16), (33, 64), (64, 64), (100, 128), (128, 128), (200, 256)])
def test_products_of_unsorted_rows(dtype, rows, tile):
    """Decode sizes: every item multiplies all rows, a tile keeps those that it holds."""
    g = torch.Generator().manual_seed(rows)
    h = torch.randn(rows, 136, generator=g).to(dtype).cuda()
    router = (torch.randn(11, 136, generator=g) * 0.1).to(dtype).cuda()
    counters = torch.zeros(12, dtype=torch.int32, device="cuda")
    order = hk.expert_select(h, router, counters, top=3, always=2, tile=tile)
    w = (torch.randn(13, 272, 136, generator=g) * 0.1).to(dtype).cuda()
    experts = torch.cat([torch.tensor([[11, 12]]).expand(rows, -1), order.chosen.cpu().long()], 1)
    products = torch.einsum("rjnk,rk->rjn", w.double().cpu()[experts], h.double().cpu())
    scores = order.scores[order.places.long()].double().cpu()[:, :, None]
    gated = oracle.silu(scores * products[..., 0::2]) * (scores * products[..., 1::2])
    for swiglu, want in ((False, products), (True, gated)):
        got = hk.grouped_linear(h, w, order, gather=True, swiglu=swiglu)[order.places.long()]
        close(got.flatten(0, 1), want.flatten(0, 1), dtype)
    kernels.runtime().check_status()


def test_choice_over_partial_sums():
    g = torch.Generator().manual_seed(0)
    parts = torch.randn(3, 70, 104, generator=g)
    counters = torch.zeros(100, dtype=torch.int32, device="cuda")
    order, _ = hk.expert_route(parts.cuda(), torch.zeros(70, 8, device="cuda"), counters, top=5, always=0, tile=32)
    want = torch.topk(parts.sum(0)[:, :99], 5, dim=-1)
    assert torch.equal(order.chosen.cpu().long(), want.indices) and torch.all(counters == 0)
    assert torch.allclose(order.chosen_scores.cpu(), torch.sigmoid(want.values), atol=1e-6)


# ------------------------------------------------------------------------ whole model ----
def small_config(variant=0):
    layers = (
        lozanex.LayerSpec("delta", DELTA[1], EXPERTS[0]),
        lozanex.LayerSpec("attention", ATTENTION[0], EXPERTS[3]),
        lozanex.LayerSpec("delta", DELTA[0], None),
        lozanex.LayerSpec("attention", dict(ATTENTION[0], mask=dict(size=31), kv_from=1), EXPERTS[2]),
        lozanex.LayerSpec("attention", ATTENTION[1], dict(EXPERTS[0], router=dict(experts=5, top=1))),
    )
    if variant == 1:
        layers = (layers[4], layers[0], layers[2])
    return lozanex.LozanexConfig(vocab_size=[101, 96][variant], hidden_size=[60, 64][variant],
                                 norm_eps=[1e-5, 1e-3][variant], layers=layers)


def decisive(config, weights):
    """Weights whose routers read dimensions that only the embedding writes, at levels well apart: no choice of
    an expert hangs on a rounding error (bf16)."""
    g = torch.Generator().manual_seed(99)
    widest = max([layer.mlp["router"]["experts"] for layer in config.layers if layer.mlp is not None], default=0)
    levels = torch.stack([torch.linspace(-2, 2, max(widest, 2))[torch.randperm(max(widest, 2), generator=g)]
                          for _ in range(config.vocab_size)])
    for name, value in weights.items():
        if name == "embed":
            value[:, :levels.shape[1]] = levels.to(value.dtype)
        elif name.endswith("embed.norm"):
            value[:levels.shape[1]] = 1.0
        elif name.endswith(("norm1", "norm2")):
            value[:widest] = 0.0
        elif name.endswith("router"):
            value.zero_()
            value.fill_diagonal_(1.0)
    return weights


def model(config, dtype, *, batch=3, capacity=256, seed=0):
    weights = decisive(config, lozanex.make_weights(config, seed=seed, dtype=dtype))
    return HybridEngine(config, cuda(weights), batch=batch, capacity=capacity), weights


def reference(config, weights, tokens, **more):
    return oracle.lozanex_forward(config.to_dict(), weights, tokens, **more)


def check_model(config, dtype, lengths, cut_lists):
    engine, weights = model(config, dtype)
    for seed, length in enumerate(lengths):
        tokens = tokens_of(config, length, seed)
        want = reference(config, weights, tokens)
        for cuts in cut_lists:
            got = run_cut(engine, tokens, cuts)
            close(got, want, dtype, MODEL_TOLERANCE[dtype])
            typical = (got.double().cpu() - want).pow(2).mean(-1).sqrt().median() / want.pow(2).mean(-1).sqrt().max()
            assert float(typical) <= TOLERANCE[dtype]


@BOTH
@pytest.mark.parametrize("variant", [0, 1])
def test_model_in_portions(dtype, variant):
    """Whole, token by token, two tokens at a time, cuts in the middle of chunks: one logit row per position."""
    check_model(small_config(variant), dtype, [140],
                [[140], [1] * 140, [2] * 70, [3, 64, 2, 66, 5], [47, 2, 15, 64, 1, 1, 10], [130, 1, 1, 1, 1, 1, 5]])


def test_model_with_undisturbed_routers():
    """fp32, where rounding does not change a choice: random routers on the whole residual stream."""
    config = small_config()
    weights = lozanex.make_weights(config, seed=5)
    engine = HybridEngine(config, cuda(weights), batch=2, capacity=128)
    tokens = tokens_of(config, 80, 3)
    want = reference(config, weights, tokens)
    for cuts in ([80], [1] * 80, [30, 2, 48]):
        close(run_cut(engine, tokens, cuts), want, torch.float32)


@BOTH
def test_residual_stream_after_every_layer(dtype):
    config = small_config()
    engine, weights = model(config, dtype)
    tokens = tokens_of(config, 40, 1)
    want, got = [], []
    reference(config, weights, tokens, streams=want)
    engine.forward([(engine.open(), tokens)], streams=got)
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
        want = reference(config, weights, tokens)
        close(run_cut(engine, tokens, [length]), want, dtype, MODEL_TOLERANCE[dtype])
        close(run_cut(engine, tokens, [1] * length), want, dtype, MODEL_TOLERANCE[dtype])


def test_equal_prompts_in_one_step_equal_each_alone():
    """Whole prompts of one length take one attention launch; slots out of order take one per sequence."""
    config = small_config()
    engine, weights = model(config, torch.bfloat16)
    prompts = [tokens_of(config, 140, s) for s in range(3)]
    want = [reference(config, weights, prompt) for prompt in prompts]
    slots = [engine.open() for _ in prompts]
    for order in (slots, slots[::-1]):
        got = engine.forward(list(zip(order, prompts)), [list(range(140))] * 3)
        for i in range(3):
            close(got[140 * i:140 * (i + 1)], want[i], torch.bfloat16, MODEL_TOLERANCE[torch.bfloat16])
        for slot in slots:
            engine.close(slot)
            assert engine.open() == slot


@BOTH
def test_unequal_batches_equal_each_alone(dtype):
    """Whole prompts, portions and decoded tokens of several sequences in one step."""
    config = small_config()
    engine, weights = model(config, dtype, batch=4)
    sequences = [tokens_of(config, n, 50 + n) for n in (90, 17, 3, 130)]
    want = [reference(config, weights, s) for s in sequences]
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


def test_slots_are_used_again():
    """A slot whose former sequence was longer gives what a fresh engine gives."""
    config = small_config()
    engine, _ = model(config, torch.bfloat16, batch=2)
    long, short = tokens_of(config, 200, 1), tokens_of(config, 33, 2)
    fresh = run_cut(engine, short, [20, 13])
    for _ in range(3):
        run_cut(engine, long, [200])
        assert torch.equal(run_cut(engine, short, [20, 13]), fresh)
    a, b = engine.open(), engine.open()
    engine.forward([(a, long[:50]), (b, short[:5])])
    engine.close(a)
    c = engine.open()
    assert c == a
    together = engine.forward([(c, short)], [list(range(33))])
    close(together, fresh.double().cpu(), torch.bfloat16, MODEL_TOLERANCE[torch.bfloat16])


@BOTH
def test_long_decoding(dtype):
    """Hundreds of decoded tokens from captured steps, through many chunks, against the whole sequence."""
    config = small_config(1)
    engine, weights = model(config, dtype, batch=2, capacity=512)
    tokens = tokens_of(config, 400, 9)
    want = reference(config, weights, tokens)
    slot = engine.open()
    engine.forward([(slot, tokens[:10])])
    for place in range(10, 400):
        engine.decode_rows([slot], [tokens[place]])
        if place % 64 in (0, 1, 63) or place == 399:  # around the chunks' edges
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
        logits = reference(config, weights, request.prompt + request.output)
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
    assert torch.equal(captured, engine.generate(prompts, 6, use_graph=False))
    scheduled, _ = model(config, torch.bfloat16, batch=3, capacity=128)
    scheduler = RequestScheduler(scheduled)
    requests = [scheduler.submit(p, 7) for p in prompts.tolist()]
    scheduler.run()
    assert [r.output for r in requests] == captured.tolist()


def test_idle_rows_leave_no_trace():
    """A decode batch rounded up with idle rows changes nothing of the slots that sit out."""
    config = small_config(1)
    engine, weights = model(config, torch.bfloat16, batch=4, capacity=64)
    slots = [engine.open() for _ in range(4)]
    prompts = [tokens_of(config, 5 + i, i) for i in range(4)]
    for slot, prompt in zip(slots, prompts):
        engine.forward([(slot, prompt)])
    before = [{k: v[slots[3]].clone() for k, v in layer.items()} for layer in engine.state.layers]
    engine.decode_rows(slots[:3], [1, 2, 3])  # four rows, one idle
    for layer, saved in zip(engine.state.layers, before):
        for name, tensor in layer.items():
            assert torch.equal(tensor[slots[3]], saved[name])
    assert engine.state.lengths.tolist() == [6, 7, 8, 8]
    for i in range(3):
        close(engine.logits[i:i + 1], reference(config, weights, prompts[i] + [i + 1])[-1:], torch.bfloat16,
              MODEL_TOLERANCE[torch.bfloat16])


# ---------------------------------------------------------------- files and command line ----
def stored_model(folder, config, seed=0):
    weights = decisive(config, lozanex.make_weights(config, seed=seed, dtype=torch.bfloat16))
    (folder / "config.json").write_text(json.dumps(config.to_dict()))
    save_safetensors(weights, folder / "model.safetensors")
    return weights


@BOTH
def test_trace_replay(dtype, tmp_path):
    """A stored model loaded through the registry and driven step by step."""
    config = small_config(1)
    weights = stored_model(tmp_path, config)
    first, second = tokens_of(config, 90, 1), tokens_of(config, 25, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": first[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": first[50:58], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": first[58:], "want": [1, 6, 0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": second, "want": [24]}], "end": ["b"]}]
    output = io.StringIO()
    engine = load_model(tmp_path, dtype=dtype, batch=1, capacity=90)
    replay(engine, [json.dumps(step) for step in steps], tmp_path, output)
    assert output.getvalue().split("\n")[:-1] == [f"done {n}" for n in range(4)]
    a, b = (reference(config, weights, t) for t in (first, second))
    for step, want in ((0, a[[0, 49]]), (2, a[[59, 64, 58]]), (3, b[[24]])):
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
