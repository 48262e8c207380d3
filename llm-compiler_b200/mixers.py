"""The sublayers of hybrid decoder layers on the sm_100a kernels: the mixers (retention, latent attention,
attention over cached keys and values, the gated delta rule with a decay per key channel or per head) and
the feed-forwards (gated MLP, mixture of experts). Each takes its sizes and constants from a spec, packs its
weights once, says what state a sequence keeps, and maps rows h to the sublayer's result for any mix of
portions and decoded tokens.

Packing: all projections of h are one stacked matrix; every operand starts at a multiple of 8 columns,
and extents are padded with zero rows / columns to multiples of 8, so that the 16-bit GEMMs take any size.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch

from . import hybrid_kernels as hk
from . import kernels
from .hybrid_kernels import SequenceBatch, Summands, pad8

ABSORBED_ROWS = 16  # longest portion that attends in the latent space (beyond: expanded keys and values)
PARTIAL_ROWS = 128  # rows up to which a projection in front of a residual leaves split-K partials


def pad_matrix(weight: torch.Tensor, rows: int, columns: int) -> torch.Tensor:
    """`weight` in the top left corner of a zero matrix."""

    if tuple(weight.shape) == (rows, columns):
        return weight.contiguous()
    padded = torch.zeros((rows, columns), dtype=weight.dtype, device=weight.device)
    padded[:weight.shape[0], :weight.shape[1]].copy_(weight)
    return padded


def stack_projections(weights: Sequence[torch.Tensor], columns: int) -> Tuple[torch.Tensor, List[int]]:
    """One [sum of padded rows, columns] matrix and the first output column of every part."""

    offsets, total = [], 0
    for weight in weights:
        offsets.append(total)
        total += pad8(weight.shape[0])
    stacked = torch.zeros((total, columns), dtype=weights[0].dtype, device=weights[0].device)
    for offset, weight in zip(offsets, weights):
        stacked[offset:offset + weight.shape[0], :weight.shape[1]].copy_(weight)
    return stacked, offsets


def block_diagonal(parts: Sequence[Tuple[torch.Tensor, int]], columns: int) -> Tuple[torch.Tensor, List[int]]:
    """Projections of neighbouring column ranges of one matrix as one GEMM: parts are (weight, first
    input column); returns the matrix and the first output column of every part."""

    stacked, offsets = stack_projections([torch.zeros((w.shape[0], 1), dtype=w.dtype, device=w.device)
                                          for w, _ in parts], columns)
    for offset, (weight, first) in zip(offsets, parts):
        stacked[offset:offset + weight.shape[0], first:first + weight.shape[1]].copy_(weight)
    return stacked, offsets


def pad_heads(weight: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    """[heads * d, k] -> [heads * size, k] with zero rows behind every head's d."""

    d = weight.shape[0] // heads
    if d == size:
        return weight
    padded = torch.zeros((heads, size, weight.shape[1]), dtype=weight.dtype, device=weight.device)
    padded[:, :d].copy_(weight.view(heads, d, -1))
    return padded.view(heads * size, -1)


def project_out(rows: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """A projection whose consumer is residual_norm: fp32 split-K partials at decode sizes (the
    consumer adds them), else the rounded result."""

    if rows.dtype == torch.bfloat16 and rows.shape[0] <= PARTIAL_ROWS:
        return kernels.b200_linear_partial(rows, weight)
    return kernels.b200_linear(rows, weight)


class Mixer:
    """One layer's mixer. `state_spec` is what a slot keeps; `shared_state` names the layer whose state
    this one reads instead of keeping its own."""

    shared_state: Optional[int] = None

    def state_spec(self, capacity: int) -> Dict[str, tuple]:
        return {}

    def __call__(self, h: torch.Tensor, batch: SequenceBatch, state: Dict[str, torch.Tensor]):
        """A tensor or Summands: what residual_norm takes."""

        raise NotImplementedError


class Retention(Mixer):
    """q, k, v and a silu gate; S' = gamma_h S + k v^T, read-out S'^T q normed per head."""

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int, heads: int, dim: int, vdim: int,
                 decay: Sequence[float], rot_dims: int, rot_base: float, epsilon: float) -> None:
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.rot_dims, self.rot_base, self.epsilon = rot_dims, rot_base, epsilon
        self.w_in, (q, k, v, self.gate_column) = stack_projections(
            [weights[name] for name in ("q", "k", "v", "g")], pad8(width))
        self.columns = (q, k, v)
        self.w_out = pad_matrix(weights["o"], pad8(width), pad8(heads * vdim))
        self.decay = torch.tensor(list(decay), dtype=torch.float32, device=self.w_in.device)
        self.k_scale = dim ** -0.5

    def state_spec(self, capacity):
        return {"state": ((self.heads, self.dim, (self.vdim + 3) // 4 * 4), torch.float32)}

    def __call__(self, h, batch, state):
        projected = kernels.b200_linear(h, self.w_in)
        inputs = hk.retention_inputs(projected, self.decay, batch, heads=self.heads, dim=self.dim, vdim=self.vdim,
                                     columns=self.columns, rot_dims=self.rot_dims, rot_base=self.rot_base,
                                     k_scale=self.k_scale)
        gate = projected[:, self.gate_column:]
        mixed = None
        if batch.decode:
            mixed = hk.recurrence_step(inputs, state["state"], gate, None, batch.sequences, kind="silu",
                                       epsilon=self.epsilon)
        if mixed is None:
            q, k, v = hk.retention_prep(inputs, h.shape[0], h.dtype, h.device)
            read_out = hk.recurrence(q, k, v, None, self.decay, state["state"], batch, h.dtype)
            mixed = hk.gated_head_norm(read_out, None, gate, kind="silu", epsilon=self.epsilon)
        return project_out(mixed, self.w_out)


class GatedDelta(Mixer):
    """Gated delta rule: short convolutions on q, k, v, unit q and k, decays from a_log, dt_bias and a
    projection of h, and a gate on the normed read-out. A subclass packs the projections and says where the
    decays (`decay_column`) and the gate (`gate_column`) stand in the matrix that `_gates` returns."""

    gate_kind: str
    decay_column: int
    gate_column: int

    def __init__(self, weights: Dict[str, torch.Tensor], *, heads: int, kv_heads: int, dim: int, vdim: int,
                 width: int, epsilon: float) -> None:
        self.heads, self.kv_heads, self.dim, self.vdim, self.epsilon = heads, kv_heads, dim, vdim, epsilon
        self.w_out = pad_matrix(weights["o"], pad8(width), pad8(heads * vdim))
        self.conv = tuple(weights[name].contiguous() for name in ("q.conv", "k.conv", "v.conv"))
        self.a_log, self.dt_bias, self.norm = weights["A_log"], weights["dt_bias"], weights["norm"]
        self.taps = self.conv[0].shape[1]
        self.q_scale = dim ** -0.5

    def state_spec(self, capacity):
        return {"state": ((self.heads, self.dim, (self.vdim + 3) // 4 * 4), torch.float32),
                "ring": ((self.taps, 2 * self.kv_heads * self.dim + self.heads * self.vdim), self.w_in.dtype)}

    def _gates(self, projected: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def __call__(self, h, batch, state):
        projected = kernels.b200_linear(h, self.w_in)
        gates = self._gates(projected)
        inputs = hk.delta_inputs(projected, gates, self.conv, self.a_log, self.dt_bias, state["ring"], batch,
                                 heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                                 columns=self.columns, decay_column=self.decay_column, q_scale=self.q_scale)
        gate = gates[:, self.gate_column:]
        mixed = None
        if batch.decode:
            mixed = hk.recurrence_step(inputs, state["state"], gate, self.norm, batch.sequences, kind=self.gate_kind,
                                       epsilon=self.epsilon)
        if mixed is None:
            q, k, v, beta, log_decay = hk.delta_prep(inputs, batch, h.dtype, h.device)
            read_out = hk.recurrence(q, k, v, beta, log_decay, state["state"], batch, h.dtype)
            hk.conv_tail(inputs, batch.sequences, h.dtype, h.device)
            mixed = hk.gated_head_norm(read_out, self.norm, gate, kind=self.gate_kind, epsilon=self.epsilon)
        return project_out(mixed, self.w_out)


class ChannelDelta(GatedDelta):
    """One decay per head and key channel, decays and a sigmoid gate from low-rank projections."""

    gate_kind = "sigmoid"

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int, **sizes) -> None:
        super().__init__(weights, width=width, **sizes)
        self.w_in, offsets = stack_projections(
            [weights[name] for name in ("q", "k", "v", "b", "a1", "g1")], pad8(width))
        self.columns = tuple(offsets[:4])
        self.low_column = offsets[4]  # a1 and g1 side by side: the input of the two up projections
        low = self.w_in.shape[0] - self.low_column
        self.w_gates, (self.decay_column, self.gate_column) = block_diagonal(
            [(weights["a2"], 0), (weights["g2"], offsets[5] - offsets[4])], low)

    def _gates(self, projected):
        return kernels.b200_linear(projected[:, self.low_column:], self.w_gates)


class HeadDelta(GatedDelta):
    """One decay per head, a full silu gate."""

    gate_kind = "silu"

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int, **sizes) -> None:
        super().__init__(weights, width=width, **sizes)
        self.w_in, offsets = stack_projections(
            [weights[name] for name in ("q", "k", "v", "b", "a", "g")], pad8(width))
        self.columns = tuple(offsets[:4])
        self.decay_column, self.gate_column = offsets[4:]

    def _gates(self, projected):
        return projected


class Attention(Mixer):
    """Grouped softmax attention over cached keys and values, with biases, RMS norms over the whole query and
    the whole key projection and a rotation of the first dimensions of every head; with `chunk` a position
    sees only its own chunk of that many positions. `kv_from` reads the caches that an earlier layer keeps."""

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int, heads: int, kv_heads: int, dim: int,
                 vdim: int, scale: float, rot_dims: int, rot_base: float, epsilon: float, chunk: Optional[int] = None,
                 kv_from: Optional[int] = None) -> None:
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.epsilon, self.chunk, self.shared_state = scale, epsilon, chunk or 0, kv_from
        names = ("q", "k", "v") if kv_from is None else ("q",)
        self.w_in, offsets = stack_projections([weights[name] for name in names], pad8(width))
        self.columns = tuple(offsets) if kv_from is None else (0, 0, 0)
        self.bias = torch.zeros(self.w_in.shape[0], dtype=self.w_in.dtype, device=self.w_in.device)
        for name, offset in zip(names, offsets):
            self.bias[offset:offset + weights[name].shape[0]].copy_(weights[name + ".b"])
        self.q_norm, self.k_norm = weights["q.norm"], weights["k.norm"] if kv_from is None else None
        # 16-bit models run on the tensor-core kernels where a head fits them: q, k and v of a head
        # zero-padded to one size of 64 or 128
        self.dense = self.w_in.dtype == torch.bfloat16 and max(dim, vdim) <= 128 and scale > 0
        self.size = (64 if max(dim, vdim) <= 64 else 128) if self.dense else pad8(max(dim, vdim))
        self.w_out = pad_matrix(pad_heads(weights["o"].t().contiguous(), heads, self.size).t(), pad8(width),
                                heads * self.size)
        self.out_bias = weights["o.b"].contiguous()
        self.turns = torch.tensor([rot_base ** (-2.0 * i / rot_dims) / (2.0 * math.pi) for i in range(rot_dims // 2)],
                                  dtype=torch.float64, device=self.w_in.device)

    def state_spec(self, capacity):
        if self.shared_state is not None:
            return {}
        row = (capacity, self.kv_heads, self.size)
        return {"keys": (row, self.w_in.dtype), "values": (row, self.w_in.dtype)}

    def __call__(self, h, batch, state):
        rows = h.shape[0]
        keys, values = state["keys"], state["values"]
        partial = h.dtype == torch.bfloat16 and rows <= PARTIAL_ROWS
        projected = kernels.b200_linear_partial(h, self.w_in) if partial else kernels.b200_linear(h, self.w_in, self.bias)
        q = hk.attention_prep(projected, self.bias if partial else None, self.q_norm, self.k_norm, self.turns, keys,
                              values, batch, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                              row_size=self.size, columns=self.columns, epsilon=self.epsilon)
        if not self.dense:
            mixed = hk.slot_attention(q, keys, values, batch, scale=self.scale, chunk=self.chunk)
        elif batch.decode:
            mixed = hk.slot_decode_attention(q, keys, values, batch, scale=self.scale, chunk=self.chunk)
        else:
            mixed = self._attend_portions(q, keys, values, batch)
        return Summands(project_out(mixed.view(rows, self.heads * self.size), self.w_out), self.out_bias)

    def _attend_portions(self, q, keys, values, batch):
        """The prefill kernel over the caches: one launch for equal whole prompts in neighbouring slots, else
        one per sequence, from the first key of the chunk that the portion starts in."""

        heads, size = q.shape[1:]
        output = torch.empty_like(q)
        slots = batch.slots_host
        if batch.uniform_start and slots == list(range(slots[0], slots[0] + len(slots))):
            groups = [(0, slots[0], len(slots), batch.counts[0], 0)]
        else:
            groups, first = [], 0
            for slot, base, count in zip(slots, batch.bases_host, batch.counts):
                groups.append((first, slot, 1, count, base))
                first += count
        for first, slot, sequences, tokens, base in groups:
            start = base // self.chunk * self.chunk if self.chunk else 0
            part = slice(first, first + sequences * tokens)
            seen = (slice(slot, slot + sequences), slice(start, base + tokens))
            hk.context_attention(q[part].view(sequences, tokens, heads, size).transpose(1, 2),
                                 keys[seen].transpose(1, 2), values[seen].transpose(1, 2), None,
                                 output[part].view(sequences, tokens, heads, size), context=base - start,
                                 scale=self.scale, chunk=self.chunk)
        return output


class LatentAttention(Mixer):
    """Attention over one cached latent per token (no rotation); `kv_from` reads the latents that
    an earlier layer keeps."""

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int, heads: int, dim: int, vdim: int,
                 q_rank: int, kv_rank: int, scale: float, epsilon: float, kv_from: Optional[int] = None) -> None:
        self.heads, self.dim, self.vdim, self.scale, self.epsilon = heads, dim, vdim, scale, epsilon
        self.q_rank, self.kv_rank, self.shared_state = q_rank, kv_rank, kv_from
        self.rank_row = (kv_rank + 15) // 16 * 16
        down = [weights["dq"]] + ([weights["dkv"]] if kv_from is None else [])
        self.w_down, offsets = stack_projections(down, pad8(width))
        self.kv_column = offsets[-1]
        self.q_norm = weights["dq.norm"]
        self.kv_norm = weights["dkv.norm"] if kv_from is None else None
        self.sink = weights["sink"].contiguous()
        self.q_size, self.v_size = pad8(dim), pad8(vdim)
        # 16-bit prompts run on the tcgen05 prefill kernel where a head fits it: q, k and v of a head
        # zero-padded to one size of 64 or 128
        self.expandable = self.w_down.dtype == torch.bfloat16 and max(dim, vdim) <= 128 and scale > 0
        if self.expandable:
            self.q_size = self.v_size = 64 if max(dim, vdim) <= 64 else 128
        self.w_q = pad_matrix(pad_heads(weights["uq"], heads, self.q_size), heads * self.q_size, pad8(q_rank))
        key = pad_heads(pad_matrix(weights["uk"], heads * dim, self.rank_row), heads, self.q_size)
        value = pad_heads(pad_matrix(weights["uv"], heads * vdim, self.rank_row), heads, self.v_size)
        self.w_into = key.view(heads, self.q_size, self.rank_row).transpose(1, 2).contiguous()
        self.w_from = value.view(heads, self.v_size, self.rank_row).contiguous()
        self.w_expand = torch.cat([key, value]).contiguous() if self.expandable else None
        out = pad_heads(weights["o"].t().contiguous(), heads, self.v_size).t()
        self.w_out = pad_matrix(out, pad8(width), heads * self.v_size)
        self.w_out = self.w_out.contiguous()

    def state_spec(self, capacity):
        if self.shared_state is not None:
            return {}
        return {"latent": ((capacity, self.rank_row), self.w_down.dtype)}

    def __call__(self, h, batch, state):
        down = kernels.b200_linear(h, self.w_down)
        cache = state["latent"]
        expand = self.expandable and batch.counts is not None and max(batch.counts) > ABSORBED_ROWS
        query_latent, dense = hk.latent_norm(down, self.q_norm, self.kv_norm, cache, batch,
                                             kv_column=self.kv_column, epsilon=self.epsilon,
                                             dense=expand and batch.uniform_start)
        if dense is not None:
            batch.dense[cache.data_ptr()] = dense
        rows = h.shape[0]
        q = kernels.b200_linear(query_latent, self.w_q).view(rows, self.heads, self.q_size)
        if expand:
            values = self._attend_expanded(q, cache, batch)
        else:
            absorbed = hk.head_linear(q, self.w_into)
            weighted = hk.latent_attention(absorbed, cache, self.sink, batch, scale=self.scale)
            values = hk.head_linear(weighted, self.w_from)
        return project_out(values.view(rows, self.heads * self.v_size), self.w_out)

    def _attend_expanded(self, q: torch.Tensor, cache: torch.Tensor, batch: SequenceBatch) -> torch.Tensor:
        """Keys and values of a portion and everything before it expanded from the latents, then the
        prefill kernel: one launch for equal whole prompts, else one per sequence."""

        rows, heads, size = q.shape
        output = torch.empty((rows, heads, size), dtype=q.dtype, device=q.device)
        dense = batch.dense.get(cache.data_ptr()) if batch.uniform_start else None
        if dense is not None:
            groups = [(0, batch.sequences, batch.counts[0], 0, dense)]
        else:
            groups, first = [], 0
            for slot, base, count in zip(batch.slots_host, batch.bases_host, batch.counts):
                groups.append((first, 1, count, base, cache[slot, :base + count]))
                first += count
        for first, sequences, tokens, context, latents in groups:
            expanded = kernels.b200_linear(latents, self.w_expand).view(sequences, context + tokens, 2 * heads, size)
            part = slice(first, first + sequences * tokens)
            hk.context_attention(q[part].view(sequences, tokens, heads, size).transpose(1, 2),
                                 expanded[:, :, :heads].transpose(1, 2), expanded[:, :, heads:].transpose(1, 2),
                                 self.sink, output[part].view(sequences, tokens, heads, size), context=context,
                                 scale=self.scale)
        return output


class GatedMlp:
    """down(silu(gate h) * (up h)): the gate and up rows interleaved for the GEMM's SwiGLU epilogue."""

    def __init__(self, weights: Dict[str, torch.Tensor], *, width: int) -> None:
        ff = pad8(weights["gate"].shape[0])
        self.w_in = kernels.interleave_gate_up(pad_matrix(weights["gate"], ff, pad8(width)),
                                               pad_matrix(weights["up"], ff, pad8(width)))
        self.w_out = pad_matrix(weights["down"], pad8(width), ff)

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return project_out(kernels.b200_linear(h, self.w_in, epilogue="swiglu"), self.w_out)


class ExpertMlp:
    """Mixture of experts: sigmoid scores of a router, the `top` best experts per token, every expert a gated
    MLP on the token scaled by its score; a shared gated MLP (None: none) runs for every token.

    A gated MLP is the sum of its slices along the feed-forward width, so at decode sizes the shared one
    runs as a few more experts of the others' size that take every token with score 1 (its weights stand
    behind theirs); for prompts it is a dense product."""

    def __init__(self, router: torch.Tensor, experts: Sequence[Dict[str, torch.Tensor]], *, width: int, top: int,
                 shared: Optional[Dict[str, torch.Tensor]] = None) -> None:
        self.top, self.experts = top, len(experts)
        self.w_router = pad_matrix(router, pad8(len(experts)), pad8(width))
        ff = pad8(experts[0]["gate"].shape[0])
        shared_ff = 0 if shared is None else pad8(shared["gate"].shape[0])
        self.slices = -(-shared_ff // ff)
        like = dict(dtype=router.dtype, device=router.device)
        self.w_in = torch.zeros((len(experts) + self.slices, 2 * ff, pad8(width)), **like)
        self.w_out = torch.zeros((len(experts) + self.slices, pad8(width), ff), **like)
        for i, expert in enumerate(experts):
            mlp = GatedMlp(expert, width=width)
            self.w_in[i].copy_(mlp.w_in)
            self.w_out[i].copy_(mlp.w_out)
        self.shared = None
        if shared is not None:
            self.shared = GatedMlp(shared, width=width)
            flat = self.w_in[len(experts):].view(-1, pad8(width))[:2 * shared_ff]
            flat.copy_(self.shared.w_in)
            self.shared.w_in = flat  # (one copy serves both forms)
            for i in range(self.slices):
                part = self.shared.w_out[:, i * ff:(i + 1) * ff]
                self.w_out[len(experts) + i, :, :part.shape[1]].copy_(part)
        self.counters = torch.zeros(len(experts) + 1, dtype=torch.int32, device=router.device)  # zero between calls

    def tile_of(self, rows: int) -> int:
        """Rows of a tile: at decode sizes every row (only those that it holds cost anything), else near the
        average number of rows an expert gets."""

        if rows <= PARTIAL_ROWS:
            return 64 if rows <= 64 else 128
        return 128 if rows * self.top <= 160 * self.experts else 256

    def __call__(self, h: torch.Tensor) -> Summands:
        rows = h.shape[0]
        tile, few = self.tile_of(rows), rows <= PARTIAL_ROWS
        ordered = h
        if few:
            order = hk.expert_select(h, self.w_router, self.counters, top=self.top, always=self.slices, tile=tile)
        else:
            logits = kernels.b200_linear_partial(h, self.w_router) if h.dtype == torch.bfloat16 \
                else kernels.b200_linear(h, self.w_router)  # (fp32 results either way)
            order, ordered = hk.expert_route(logits, h, self.counters, top=self.top, always=0, tile=tile)
        inner = hk.grouped_linear(ordered, self.w_in, order, gather=few, swiglu=True)
        return Summands(None if few or self.shared is None else self.shared(h), None,
                        hk.grouped_linear(inner, self.w_out, order), order.places)


@dataclass
class HybridLayer:
    """What HybridEngine runs: a mixer and a feed-forward (or none), a norm behind each and, in designs whose
    sublayers do not read the residual itself, one in front of each."""

    mixer: Mixer
    norm_in: Optional[torch.Tensor]
    norm_out: torch.Tensor
    mlp: Optional[Callable[[torch.Tensor], object]] = None
    mlp_norm_in: Optional[torch.Tensor] = None
    mlp_norm_out: Optional[torch.Tensor] = None
