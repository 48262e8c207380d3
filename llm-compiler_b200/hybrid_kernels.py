"""Python wrappers over the C ABI for the hybrid layers' operators (include/b200_serve.h, "Hybrid
layers"): recurrent mixers, attention over cached latents or keys and values, mixtures of experts and the
fp32 residual stream. Same rules as kernels.py:
preconditions raise before anything is launched, launches go to torch's current stream and never
synchronise, and there is no fallback to PyTorch."""

from __future__ import annotations

from ctypes import byref
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

import torch

from . import _lib
from .kernels import _check, _code, _count, _ptr, _require_cuda, _stream, runtime

CHUNK = 64  # tokens of a chunk of recurrence_chunked
CHUNKED_FROM = 24  # longest portion of a step from which the chunked form is the faster one
GATES = {"silu": _lib.GATE_SILU, "sigmoid": _lib.GATE_SIGMOID}


def pad8(extent: int) -> int:
    """Row strides and GEMM extents of 16-bit operands are multiples of 8 elements (16 bytes)."""

    return (extent + 7) // 8 * 8


@dataclass
class SequenceBatch:
    """The rows of a step as sequences: `rows` tokens of `sequences` sequences, and the four device
    vectors of the header's description. `counts` / `bases_host` are the host's copy of the portion
    lengths and first positions (None inside a captured decode step, where every count is 1)."""

    rows: int
    sequences: int
    token_sequence: torch.Tensor
    starts: torch.Tensor
    slots: torch.Tensor
    bases: torch.Tensor
    counts: Optional[List[int]] = None
    bases_host: Optional[List[int]] = None
    slots_host: Optional[List[int]] = None
    dense: dict = field(default_factory=dict)  # layer state -> this step's latents side by side
    _chunks: Optional[Tuple[torch.Tensor, int]] = None

    @property
    def decode(self) -> bool:
        return self.counts is None or max(self.counts) == 1

    @property
    def uniform_start(self) -> bool:
        """Every portion starts its sequence and all are of one length."""

        return self.counts is not None and not any(self.bases_host) and len(set(self.counts)) == 1

    def chunk_table(self) -> Tuple[torch.Tensor, int]:
        """First chunk of every sequence (int32 [sequences + 1]) and the number of chunks."""

        if self._chunks is None:
            table = [0]
            for count in self.counts:
                table.append(table[-1] + -(-count // CHUNK))
            self._chunks = (torch.tensor(table, dtype=torch.int32).to(self.starts.device), table[-1])
        return self._chunks

    @property
    def longest(self) -> int:
        return 1 if self.counts is None else max(self.counts)

    def context_bound(self, capacity: int) -> int:
        """Upper bound of the positions any row of this step sees."""

        if self.counts is None:
            return capacity
        return min(capacity, max(base + count for base, count in zip(self.bases_host, self.counts)))

    def pointers(self) -> Tuple[int, int, int, int]:
        return (self.token_sequence.data_ptr(), self.starts.data_ptr(), self.slots.data_ptr(),
                self.bases.data_ptr())


def _require_rows(tensor: torch.Tensor, what: str) -> None:
    if tensor.ndim != 2 or tensor.stride(1) != 1:
        raise ValueError(f"{what} must be a matrix with contiguous rows")


@dataclass
class Summands:
    """A sublayer's result in the parts that residual_norm adds up: y (as there) plus `bias` [width], and
    for every row the rows `places` [rows, top] of the matrix `rows` (the experts' results)."""

    y: Optional[torch.Tensor]
    bias: Optional[torch.Tensor] = None
    rows: Optional[torch.Tensor] = None
    places: Optional[torch.Tensor] = None


def embedding_residual(table: torch.Tensor, ids: torch.Tensor, weight: Optional[torch.Tensor] = None, *,
                       epsilon: float = 0.0, weight_offset: float = 0.0, narrow: bool = False):
    """Rows of `table` gathered by int64 ids and widened to fp32: the start of the residual stream. With
    `weight` the rows are normed and scaled by weight_offset + weight; with `narrow` also returns them in
    the table's dtype (padded to 8 elements)."""

    device = _require_cuda(table, ids, weight)
    if table.ndim != 2 or not table.is_contiguous() or ids.dtype != torch.int64 or ids.ndim != 1 or \
            not ids.is_contiguous():
        raise ValueError("embedding needs a contiguous V x H table and a vector of int64 ids")
    if weight is not None and (weight.shape != (table.shape[1],) or weight.dtype != table.dtype):
        raise ValueError("the norm weight must be a vector of the table's width")
    x = torch.empty((ids.shape[0], table.shape[1]), dtype=torch.float32, device=device)
    h = torch.empty((ids.shape[0], pad8(table.shape[1])), dtype=table.dtype, device=device) if narrow else None
    rt = runtime(device)
    code = _lib.load().b200_embedding_residual(table.data_ptr(), _ptr(weight), ids.data_ptr(), x.data_ptr(), _ptr(h),
                                               ids.shape[0], table.shape[1], table.shape[0], pad8(table.shape[1]),
                                               float(epsilon), float(weight_offset), _code(table.dtype),
                                               rt.status.data_ptr(), _stream())
    _check(code, "b200_embedding_residual")
    _count(rt)
    return (x, h) if narrow else x


def residual_norm(x: torch.Tensor, y, post_weight: Optional[torch.Tensor],
                  next_weight: Optional[torch.Tensor], *, epsilon: float, weight_offset: float,
                  dtype: torch.dtype, narrow: bool = False) -> Optional[torch.Tensor]:
    """x += norm(y) * (weight_offset + post_weight) in place on the fp32 residual x [rows, width], then
    h = norm(x) * (weight_offset + next_weight), returned in `dtype` with rows padded to 8 elements; without
    next_weight h is x itself (narrow) or nothing. y: [rows, >= width] in `dtype`, fp32 split-K partials
    [splits, rows, >= width], or Summands; None: h only."""

    parts = y if isinstance(y, Summands) else Summands(y)
    y = parts.y
    device = _require_cuda(x, y, post_weight, next_weight, parts.bias, parts.rows, parts.places)
    if x.ndim != 2 or x.dtype != torch.float32 or not x.is_contiguous():
        raise ValueError("the residual is a contiguous fp32 matrix")
    rows, width = x.shape
    splits = y_stride = top = summand_stride = 0
    if y is not None:
        if y.ndim == 3:
            if y.dtype != torch.float32 or not y.is_contiguous() or y.shape[1] != rows:
                raise ValueError("partial sums must be a contiguous fp32 [splits, rows, columns] tensor")
            splits, y_stride = y.shape[0], y.shape[2]
        else:
            _require_rows(y, "the sublayer's result")
            if y.dtype != dtype or y.shape[0] != rows:
                raise ValueError("the sublayer's result does not match the residual")
            y_stride = y.stride(0)
        if y.shape[-1] < width:
            raise ValueError("the sublayer's result is narrower than the residual")
    if parts.rows is not None:
        _require_rows(parts.rows, "the summands")
        if parts.rows.dtype != dtype or parts.rows.shape[1] < width or parts.places is None or \
                parts.places.dtype != torch.int32 or parts.places.shape[0] != rows or not parts.places.is_contiguous():
            raise ValueError("summands must be rows of the residual's width with int32 places for every row")
        top, summand_stride = parts.places.shape[1], parts.rows.stride(0)
    if parts.bias is not None and (parts.bias.shape[0] < width or parts.bias.dtype != dtype):
        raise ValueError("the bias must be a vector of the residual's width")
    if (y is not None or top) and (post_weight is None or post_weight.shape != (width,) or post_weight.dtype != dtype):
        raise ValueError("the norm behind a sublayer needs a weight and a result of the residual's width")
    h = None
    if next_weight is not None or narrow:
        if next_weight is not None and (next_weight.shape != (width,) or next_weight.dtype != dtype):
            raise ValueError("the norm weight must be a vector of the residual's width")
        h = torch.empty((rows, pad8(width)), dtype=dtype, device=device)
    rt = runtime(device)
    code = _lib.load().b200_residual_norm(
        x.data_ptr(), _ptr(y), _ptr(parts.bias), _ptr(post_weight), _ptr(next_weight), _ptr(h), _ptr(parts.rows),
        _ptr(parts.places), rows, width, splits, top, y_stride, pad8(width), summand_stride, float(epsilon),
        float(weight_offset), _code(dtype), _stream())
    _check(code, "b200_residual_norm")
    _count(rt)
    return h


def latent_norm(projected: torch.Tensor, q_weight: torch.Tensor, kv_weight: Optional[torch.Tensor],
                cache: Optional[torch.Tensor], batch: SequenceBatch, *, kv_column: int, epsilon: float,
                dense: bool = False) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """RMS norms of the query latent (column 0 of `projected`) and, with kv_weight, of the kv latent
    (from kv_column), which is stored in the cache [slots, capacity, row] at the tokens' positions.
    Returns the query latent (rows padded to 8 elements) and, with dense, the kv latents [rows, row]."""

    device = _require_cuda(projected, q_weight, kv_weight, cache)
    _require_rows(projected, "the projection")
    q_rank = q_weight.shape[0]
    rows = projected.shape[0]
    if projected.dtype != q_weight.dtype or (kv_weight is not None and (
            cache is None or cache.dtype != projected.dtype or not cache.is_contiguous())):
        raise ValueError("projection, weights and cache must share one dtype")
    q_out = torch.empty((rows, pad8(q_rank)), dtype=projected.dtype, device=device)
    kv_rank = kv_weight.shape[0] if kv_weight is not None else 0
    row = cache.shape[2] if kv_weight is not None else 0
    dense_out = torch.empty((rows, row), dtype=projected.dtype, device=device) \
        if dense and kv_weight is not None else None
    rt = runtime(device)
    code = _lib.load().b200_latent_norm(
        projected.data_ptr(), q_weight.data_ptr(), _ptr(kv_weight), q_out.data_ptr(),
        _ptr(cache) if kv_weight is not None else None, _ptr(dense_out), *batch.pointers(), rows, q_rank, kv_rank,
        kv_column, row, projected.stride(0), q_out.stride(0), cache.shape[1] if kv_weight is not None else 0,
        float(epsilon), _code(projected.dtype), rt.status.data_ptr(), _stream())
    _check(code, "b200_latent_norm")
    _count(rt)
    return q_out, dense_out


def gated_head_norm(read_out: torch.Tensor, weight: Optional[torch.Tensor], gate: torch.Tensor, *, kind: str,
                    epsilon: float) -> torch.Tensor:
    """Per-head RMS norm of a read-out (fp32 [rows, heads, vdim]) times `weight` and silu or sigmoid of
    `gate` [rows, >= heads * vdim]; rows of the result are padded to 8 elements."""

    device = _require_cuda(read_out, weight, gate)
    rows, heads, vdim = read_out.shape
    _require_rows(gate, "the gate")
    if read_out.dtype != torch.float32 or not read_out.is_contiguous() or gate.shape[0] != rows:
        raise ValueError("the read-out must be contiguous fp32 and match the gate")
    output = torch.empty((rows, pad8(heads * vdim)), dtype=gate.dtype, device=device)
    rt = runtime(device)
    code = _lib.load().b200_gated_head_norm(
        read_out.data_ptr(), _ptr(weight), gate.data_ptr(), output.data_ptr(), rows, heads, vdim, gate.stride(0),
        output.stride(0), GATES[kind], float(epsilon), _code(gate.dtype), _stream())
    _check(code, "b200_gated_head_norm")
    _count(rt)
    return output


def retention_inputs(projected: torch.Tensor, decay: torch.Tensor, batch: SequenceBatch, *, heads: int, dim: int,
                     vdim: int, columns: Tuple[int, int, int], rot_dims: int, rot_base: float,
                     k_scale: float) -> "_lib.RetentionInputs":
    """The argument block of the retention kernels: the columns (q, k, v) of the projections, the
    rotation and the decay of every head."""

    _require_cuda(projected, decay)
    _require_rows(projected, "the projection")
    if decay.dtype != torch.float32 or decay.shape != (heads,):
        raise ValueError("retention needs one fp32 decay per head")
    inputs = _lib.RetentionInputs(projected.data_ptr(), decay.data_ptr(), *batch.pointers(), heads, dim, vdim,
                                  *columns, projected.stride(0), rot_dims, float(rot_base), float(k_scale))
    inputs.tensors = (projected, decay, batch)  # alive as long as the block that points into them
    return inputs


def retention_prep(inputs: "_lib.RetentionInputs", rows: int, dtype: torch.dtype, device: torch.device):
    """fp32 operands q, k [rows, heads, dim] (rotated, k scaled) and v [rows, heads, vdim]."""

    q = torch.empty((rows, inputs.heads, inputs.dim), dtype=torch.float32, device=device)
    k = torch.empty_like(q)
    v = torch.empty((rows, inputs.heads, inputs.vdim), dtype=torch.float32, device=device)
    rt = runtime(device)
    _check(_lib.load().b200_retention_prep(byref(inputs), q.data_ptr(), k.data_ptr(), v.data_ptr(), rows,
                                           _code(dtype), _stream()), "b200_retention_prep")
    _count(rt)
    return q, k, v


def recurrence_step(inputs, state: torch.Tensor, gate: torch.Tensor, weight: Optional[torch.Tensor],
                    sequences: int, *, kind: str, epsilon: float) -> Optional[torch.Tensor]:
    """Decode step of a recurrent mixer in one launch (inputs: retention_inputs or delta_inputs): state
    update, read-out, per-head norm and gate. Returns [sequences, heads * vdim padded to 8], or None
    where the state of a head is too large for the fused kernel."""

    device = _require_cuda(state, gate, weight)
    _require_rows(gate, "the gate")
    if state.dtype != torch.float32 or state.ndim != 4 or not state.is_contiguous() or \
            state.shape[1] != inputs.heads or state.shape[2] != inputs.dim or state.shape[3] < inputs.vdim:
        raise ValueError("the state must be contiguous fp32 [slots, heads, dim, >= vdim]")
    output = torch.empty((sequences, pad8(inputs.heads * inputs.vdim)), dtype=gate.dtype, device=device)
    block = _lib.StepOutput(state.data_ptr(), gate.data_ptr(), _ptr(weight), output.data_ptr(), state.shape[3],
                            gate.stride(0), output.stride(0), GATES[kind], float(epsilon))
    rt = runtime(device)
    call = _lib.load().b200_delta_step if isinstance(inputs, _lib.DeltaInputs) else _lib.load().b200_retention_step
    code = call(byref(inputs), byref(block), sequences, _code(gate.dtype), _stream())
    if code == _lib.ERR_UNSUPPORTED:
        return None
    _check(code, "recurrence step")
    _count(rt)
    return output


def delta_inputs(projected: torch.Tensor, gates: torch.Tensor, conv: Tuple[torch.Tensor, torch.Tensor, torch.Tensor],
                 a_log: torch.Tensor, dt_bias: torch.Tensor, ring: torch.Tensor, batch: SequenceBatch, *,
                 heads: int, kv_heads: int, dim: int, vdim: int, columns: Tuple[int, int, int, int],
                 decay_column: int, q_scale: float) -> "_lib.DeltaInputs":
    """The argument block of the gated delta rule's kernels: projections (columns of q, k, v and beta),
    decay projections, convolution taps, and the ring of earlier inputs [slots, taps, channels]. dt_bias has
    heads * dim elements (a decay per key channel) or heads (one per head)."""

    _require_cuda(projected, gates, *conv, a_log, dt_bias, ring)
    _require_rows(projected, "the projection")
    _require_rows(gates, "the gate projection")
    taps = conv[0].shape[1]
    if ring.shape[1:] != (taps, 2 * kv_heads * dim + heads * vdim) or not ring.is_contiguous():
        raise ValueError("the ring must hold `taps` inputs of every channel")
    if len({t.dtype for t in (projected, gates, *conv, a_log, dt_bias, ring)}) != 1:
        raise ValueError("projections, weights and ring must share one dtype")
    if dt_bias.numel() not in (heads, heads * dim):
        raise ValueError("decays are per head or per key channel")
    inputs = _lib.DeltaInputs(
        projected.data_ptr(), gates.data_ptr(), conv[0].data_ptr(), conv[1].data_ptr(), conv[2].data_ptr(),
        a_log.data_ptr(), dt_bias.data_ptr(), ring.data_ptr(), *batch.pointers(), heads, kv_heads, dim, vdim, taps,
        *columns, decay_column, projected.stride(0), gates.stride(0), dt_bias.numel() // heads, float(q_scale))
    inputs.tensors = (projected, gates, conv, a_log, dt_bias, ring, batch)
    return inputs


def delta_prep(inputs: "_lib.DeltaInputs", batch: SequenceBatch, dtype: torch.dtype, device: torch.device):
    """fp32 operands of the gated delta rule: q, k [rows, kv_heads, dim], v [rows, heads, vdim],
    beta [rows, heads] and log g [rows, heads, dim or 1]."""

    rows = batch.rows
    q = torch.empty((rows, inputs.kv_heads, inputs.dim), dtype=torch.float32, device=device)
    k = torch.empty_like(q)
    v = torch.empty((rows, inputs.heads, inputs.vdim), dtype=torch.float32, device=device)
    beta = torch.empty((rows, inputs.heads), dtype=torch.float32, device=device)
    decay = torch.empty((rows, inputs.heads, inputs.decay_dim), dtype=torch.float32, device=device)
    rt = runtime(device)
    code = _lib.load().b200_delta_prep(byref(inputs), q.data_ptr(), k.data_ptr(), v.data_ptr(), beta.data_ptr(),
                                       decay.data_ptr(), rows, batch.sequences, batch.longest, _code(dtype), _stream())
    _check(code, "b200_delta_prep")
    _count(rt)
    return q, k, v, beta, decay


def conv_tail(inputs: "_lib.DeltaInputs", sequences: int, dtype: torch.dtype, device: torch.device) -> None:
    """Keeps every sequence's last inputs for the short convolution of its next portion."""

    rt = runtime(device)
    _check(_lib.load().b200_conv_tail(byref(inputs), sequences, _code(dtype), _stream()), "b200_conv_tail")
    _count(rt)


def recurrence_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: Optional[torch.Tensor],
                    decay: torch.Tensor, state: torch.Tensor, batch: SequenceBatch) -> torch.Tensor:
    """Token by token recurrence over prepared fp32 operands; state [slots, heads, dim, row] is updated
    in place. beta None: retention with `decay` [heads]; else the delta rule, `decay` is log g
    [rows, heads, dim or 1]. Returns the read-out [rows, heads, vdim]."""

    device = _require_cuda(q, k, v, beta, decay, state)
    rows, kv_heads, dim = q.shape
    heads, vdim = v.shape[1], v.shape[2]
    if state.dtype != torch.float32 or state.ndim != 4 or not state.is_contiguous() or \
            state.shape[1] != heads or state.shape[2] != dim or state.shape[3] < vdim:
        raise ValueError("the state must be contiguous fp32 [slots, heads, dim, >= vdim]")
    output = torch.empty((rows, heads, vdim), dtype=torch.float32, device=device)
    rt = runtime(device)
    code = _lib.load().b200_recurrence_scan(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), _ptr(beta), decay.data_ptr(), state.data_ptr(), output.data_ptr(),
        *batch.pointers(), batch.sequences, heads, kv_heads, dim, vdim, state.shape[3],
        dim if beta is None else decay.shape[2], _stream())
    _check(code, "b200_recurrence_scan")
    _count(rt)
    return output


def recurrence_chunked(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: Optional[torch.Tensor],
                       decay: torch.Tensor, state: torch.Tensor, batch: SequenceBatch) -> Optional[torch.Tensor]:
    """recurrence_scan in chunks of 64 tokens on the tensor cores; None where the sizes do not fit."""

    device = _require_cuda(q, k, v, beta, decay, state)
    rows, kv_heads, dim = q.shape
    heads, vdim = v.shape[1], v.shape[2]
    if state.dtype != torch.float32 or state.ndim != 4 or not state.is_contiguous() or \
            state.shape[1] != heads or state.shape[2] != dim or state.shape[3] < vdim:
        raise ValueError("the state must be contiguous fp32 [slots, heads, dim, >= vdim]")
    library = _lib.load()
    starts, chunks = batch.chunk_table()
    need = int(library.b200_recurrence_chunked_workspace_bytes(chunks, heads, dim, vdim, int(beta is not None)))
    if need == 0:
        return None
    output = torch.empty((rows, heads, vdim), dtype=torch.float32, device=device)
    rt = runtime(device)
    workspace = rt.workspace("recurrence_chunked", need)
    code = library.b200_recurrence_chunked(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), _ptr(beta), decay.data_ptr(), state.data_ptr(), output.data_ptr(),
        *batch.pointers(), starts.data_ptr(), chunks, batch.sequences, heads, kv_heads, dim, vdim, state.shape[3],
        dim if beta is None else decay.shape[2], _ptr(workspace), need, _stream())
    _check(code, "b200_recurrence_chunked")
    _count(rt, 2)
    return output


def recurrence(q, k, v, beta, decay, state, batch: SequenceBatch, dtype: torch.dtype) -> torch.Tensor:
    """The recurrence over a step's portions: chunked for prompts of 16-bit models, else token by token."""

    output = None
    if dtype == torch.bfloat16 and batch.counts is not None and max(batch.counts) >= CHUNKED_FROM:
        output = recurrence_chunked(q, k, v, beta, decay, state, batch)
    return recurrence_scan(q, k, v, beta, decay, state, batch) if output is None else output


def head_linear(x: torch.Tensor, weight: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y[m, h, :] = weight[h] x[m, h, :]: x [rows, heads, k] (last dimension contiguous), weight
    [heads, n, k]. `out` may be a [rows, heads, n] view of a wider matrix."""

    device = _require_cuda(x, weight, out)
    rows, heads, k = x.shape
    if weight.ndim != 3 or weight.shape[0] != heads or weight.shape[2] != k or not weight.is_contiguous() or \
            weight.dtype != x.dtype or x.stride(2) != 1:
        raise ValueError("head_linear needs x [rows, heads, k] and a contiguous weight [heads, n, k]")
    n = weight.shape[1]
    if out is None:
        out = torch.empty((rows, heads, n), dtype=x.dtype, device=device)
    rt = runtime(device)
    code = _lib.load().b200_head_linear(x.data_ptr(), weight.data_ptr(), out.data_ptr(), rows, heads, k, n,
                                        x.stride(0), x.stride(1), out.stride(0), out.stride(1), _code(x.dtype),
                                        _stream())
    _check(code, "b200_head_linear")
    _count(rt)
    return out


def latent_attention(q: torch.Tensor, cache: torch.Tensor, sink: Optional[torch.Tensor], batch: SequenceBatch, *,
                     scale: float) -> torch.Tensor:
    """Attention of queries in the latent space [rows, heads, row] over the cached latents [slots,
    capacity, row] of their sequences; returns the weighted latents [rows, heads, row]."""

    device = _require_cuda(q, cache, sink)
    rows, heads, row = q.shape
    if not q.is_contiguous() or not cache.is_contiguous() or cache.shape[2] != row or cache.dtype != q.dtype:
        raise ValueError("queries and cached latents must be contiguous and of one row size and dtype")
    output = torch.empty_like(q)
    rt = runtime(device)
    library = _lib.load()
    longest = batch.longest
    context = batch.context_bound(cache.shape[1])
    need = int(library.b200_latent_attention_workspace_bytes(rows, batch.sequences, longest, heads, row, context,
                                                            _code(q.dtype)))
    workspace = rt.workspace("latent_attention", need)
    code = library.b200_latent_attention(
        q.data_ptr(), cache.data_ptr(), _ptr(sink), output.data_ptr(), *batch.pointers(), rows, batch.sequences,
        longest, heads, row, cache.shape[0], cache.shape[1], context, float(scale), _code(q.dtype), _ptr(workspace),
        need, rt.status.data_ptr(), _stream())
    _check(code, "b200_latent_attention")
    _count(rt, 2 if need else 1)
    return output


def context_attention(query: torch.Tensor, key: torch.Tensor, value: torch.Tensor, sink: Optional[torch.Tensor],
                      output: torch.Tensor, *, context: int, scale: float, chunk: int = 0) -> None:
    """Causal attention of a portion on the tcgen05 prefill kernel: query B x H x T x D behind `context`
    earlier positions, key / value B x Hkv x (context + T) x D (views), output memory B x T x H x D. With
    `chunk` a position sees only its own chunk of that many positions, counted from key 0."""

    device = _require_cuda(query, key, value, sink, output)
    batch, heads, tokens, dim = query.shape
    if key.shape != value.shape or key.shape[2] != context + tokens or key.shape[3] != dim:
        raise ValueError("keys and values must hold the context and the portion")
    if output.shape != (batch, tokens, heads, dim) or not output.is_contiguous():
        raise ValueError("output must be a contiguous B x T x H x D tensor")
    rt = runtime(device)
    code = _lib.load().b200_context_attention(
        query.data_ptr(), key.data_ptr(), value.data_ptr(), _ptr(sink), output.data_ptr(), batch, heads, key.shape[1],
        tokens, context, chunk, dim, _lib.i64_array(query.stride()), _lib.i64_array(key.stride()),
        _lib.i64_array(value.stride()), float(scale), rt.status.data_ptr(), _stream())
    _check(code, "b200_context_attention")
    _count(rt)


def attention_prep(projected: torch.Tensor, bias: Optional[torch.Tensor], q_weight: torch.Tensor,
                   k_weight: Optional[torch.Tensor], turns: torch.Tensor, keys: Optional[torch.Tensor],
                   values: Optional[torch.Tensor], batch: SequenceBatch, *, heads: int, kv_heads: int, dim: int,
                   vdim: int, row_size: int, columns: Tuple[int, int, int], epsilon: float) -> torch.Tensor:
    """Queries [rows, heads, row_size] of a stacked projection (columns: where q, k and v start), normed over
    the whole projection and rotated; with k_weight, keys and values go to the caches [slots, capacity,
    kv_heads, row_size]. projected: [rows, columns], or fp32 partials [splits, rows, columns] to which `bias`
    is added. turns (fp64): turns per position of every rotated pair."""

    device = _require_cuda(projected, bias, q_weight, k_weight, turns, keys, values)
    partial = projected.ndim == 3
    rows = projected.shape[-2]
    if partial:
        if projected.dtype != torch.float32 or not projected.is_contiguous():
            raise ValueError("partial sums must be a contiguous fp32 [splits, rows, columns] tensor")
    else:
        _require_rows(projected, "the projection")
        if projected.dtype != q_weight.dtype or bias is not None:
            raise ValueError("a finished projection has the weights' dtype and its bias")
    if turns.dtype != torch.float64 or q_weight.shape != (heads * dim,):
        raise ValueError("turns are fp64, the query norm's weight spans the projection")
    if k_weight is not None and (keys is None or values is None or keys.shape != values.shape or
                                 keys.shape[2:] != (kv_heads, row_size) or keys.dtype != q_weight.dtype or
                                 k_weight.shape != (kv_heads * dim,) or
                                 not (keys.is_contiguous() and values.is_contiguous())):
        raise ValueError("caches must be contiguous [slots, capacity, kv_heads, row_size] in the weights' dtype")
    own = k_weight is not None
    q = torch.empty((rows, heads, row_size), dtype=q_weight.dtype, device=device)
    inputs = _lib.AttentionPrepInputs(
        projected.data_ptr(), _ptr(bias), q_weight.data_ptr(), _ptr(k_weight), turns.data_ptr(), q.data_ptr(),
        _ptr(keys) if own else None, _ptr(values) if own else None, *batch.pointers(), rows, heads, kv_heads, dim, vdim,
        row_size, 2 * turns.shape[0], *columns, projected.stride(-2), projected.shape[0] if partial else 0,
        keys.shape[1] if own else 0, float(epsilon))
    rt = runtime(device)
    _check(_lib.load().b200_attention_prep(byref(inputs), _code(q_weight.dtype), rt.status.data_ptr(), _stream()),
           "b200_attention_prep")
    _count(rt)
    return q


def _check_caches(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor) -> None:
    if not (q.is_contiguous() and keys.is_contiguous() and values.is_contiguous()) or q.ndim != 3 or \
            keys.shape != values.shape or keys.shape[3] != q.shape[2] or len({q.dtype, keys.dtype, values.dtype}) != 1 or \
            q.shape[1] % keys.shape[2]:
        raise ValueError("queries [rows, heads, size] and caches [slots, capacity, kv_heads, size] must fit")


def slot_decode_attention(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, batch: SequenceBatch, *,
                          scale: float, chunk: int = 0) -> torch.Tensor:
    """Attention of one token per sequence over its slot's cache (bf16, rows of 64 or 128), with `chunk`
    over the token's own chunk of positions; returns [rows, heads, size]."""

    device = _require_cuda(q, keys, values)
    _check_caches(q, keys, values)
    rows, heads, size = q.shape
    if rows != batch.sequences or q.dtype != torch.bfloat16:
        raise ValueError("decode attention takes one bf16 row per sequence")
    context = batch.context_bound(keys.shape[1])
    if chunk:
        context = min(context, chunk)
    output = torch.empty_like(q)
    rt = runtime(device)
    library = _lib.load()
    need = int(library.b200_slot_decode_attention_workspace_bytes(rows, heads, keys.shape[2], size, context))
    workspace = rt.workspace("decode_attention", need)
    code = library.b200_slot_decode_attention(
        q.data_ptr(), keys.data_ptr(), values.data_ptr(), output.data_ptr(), batch.slots.data_ptr(),
        batch.bases.data_ptr(), rows, heads, keys.shape[2], size, keys.shape[0], keys.shape[1], chunk, context,
        float(scale), _ptr(workspace), need, rt.status.data_ptr(), _stream())
    _check(code, "b200_slot_decode_attention")
    _count(rt)
    return output


def slot_attention(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, batch: SequenceBatch, *,
                   scale: float, chunk: int = 0) -> torch.Tensor:
    """The same for any rows, sizes and dtype, on the CUDA cores."""

    device = _require_cuda(q, keys, values)
    _check_caches(q, keys, values)
    rows, heads, size = q.shape
    output = torch.empty_like(q)
    rt = runtime(device)
    code = _lib.load().b200_slot_attention(
        q.data_ptr(), keys.data_ptr(), values.data_ptr(), output.data_ptr(), *batch.pointers(), rows, heads,
        keys.shape[2], size, keys.shape[1], chunk, float(scale), _code(q.dtype), _stream())
    _check(code, "b200_slot_attention")
    _count(rt)
    return output


@dataclass
class ExpertOrder:
    """The rows of a step in the order of the experts they go to: for every sorted row its row (`index`) and
    score, the table of tiles (expert, rows held) and, for every row, its sorted rows (`places`)."""

    index: torch.Tensor
    scores: torch.Tensor
    tiles: torch.Tensor
    places: torch.Tensor
    tile: int
    chosen: torch.Tensor  # [rows, top]
    chosen_scores: torch.Tensor


def _expert_order(rows: int, counters: torch.Tensor, top: int, always: int, tile: int):
    experts, device = counters.shape[0] - 1, counters.device
    if counters.dtype != torch.int32 or not 0 < top <= experts:
        raise ValueError("a row takes some of the experts; counters are int32 [experts + 1]")
    max_tiles = always * -(-rows // tile) + rows * top // tile + min(experts, rows * top)
    int32 = dict(dtype=torch.int32, device=device)
    order = ExpertOrder(torch.empty(max_tiles * tile, **int32),
                        torch.empty(max_tiles * tile, dtype=torch.float32, device=device),
                        torch.empty((max_tiles, 2), **int32), torch.empty((rows, always + top), **int32), tile,
                        torch.empty((rows, top), **int32), torch.empty((rows, top), dtype=torch.float32, device=device))
    numbers = torch.empty((rows, top), **int32)
    block = _lib.ExpertOrder(order.chosen.data_ptr(), order.chosen_scores.data_ptr(), numbers.data_ptr(),
                             counters.data_ptr(), order.places.data_ptr(), order.index.data_ptr(),
                             order.scores.data_ptr(), order.tiles.data_ptr(), experts, top, always, tile, max_tiles)
    block.tensors = (order, numbers, counters)
    return order, block


def expert_select(h: torch.Tensor, router: torch.Tensor, counters: torch.Tensor, *, top: int, always: int,
                  tile: int) -> ExpertOrder:
    """The `top` experts of a few rows h by the router [>= experts, columns of h], in one launch. `always`
    more experts, numbered behind the others, take every row with score 1. counters: int32 [experts + 1],
    zero, and zero again behind the call."""

    device = _require_cuda(h, router, counters)
    _require_rows(h, "the rows")
    if router.shape[1] != h.shape[1] or router.shape[0] < counters.shape[0] - 1 or router.dtype != h.dtype or \
            not router.is_contiguous():
        raise ValueError("the router needs a contiguous row of h's columns for every expert")
    order, block = _expert_order(h.shape[0], counters, top, always, tile)
    rt = runtime(device)
    _check(_lib.load().b200_expert_select(h.data_ptr(), router.data_ptr(), byref(block), h.shape[0], h.shape[1],
                                          h.stride(0), _code(h.dtype), _stream()), "b200_expert_select")
    _count(rt)
    return order


def expert_route(logits: torch.Tensor, h: torch.Tensor, counters: torch.Tensor, *, top: int, always: int,
                 tile: int) -> Tuple[ExpertOrder, torch.Tensor]:
    """The same for many rows from finished logits: fp32 [rows, >= experts] or split-K partials of them. Also
    returns the rows of h in their order."""

    device = _require_cuda(logits, h, counters)
    _require_rows(h, "the rows")
    rows = logits.shape[-2]
    if logits.dtype != torch.float32 or not logits.is_contiguous() or h.shape[0] != rows:
        raise ValueError("the router's logits are contiguous fp32, a row for every row of h")
    order, block = _expert_order(rows, counters, top, always, tile)
    ordered = torch.empty((order.index.shape[0], h.shape[1]), dtype=h.dtype, device=device)
    rt = runtime(device)
    library = _lib.load()
    _check(library.b200_expert_route(logits.data_ptr(), byref(block), rows, logits.shape[0] if logits.ndim == 3 else 1,
                                     logits.shape[-1], _stream()), "b200_expert_route")
    _check(library.b200_expert_place(byref(block), h.data_ptr(), ordered.data_ptr(), rows, h.shape[1], h.stride(0),
                                     _code(h.dtype), _stream()), "b200_expert_place")
    _count(rt, 2)
    return order, ordered


def grouped_linear(x: torch.Tensor, weight: torch.Tensor, order: ExpertOrder, *, gather: bool = False,
                   swiglu: bool = False) -> torch.Tensor:
    """out[r] = weight[expert of r] x[r] over sorted rows; weight [experts, n, k]. gather: x holds the step's
    rows themselves, not sorted (at most `order.tile` of them). swiglu: the rows of a weight alternate gate and up, and the result is
    silu(s gate) * (s up) with the row's score s."""

    device = _require_cuda(x, weight, order.tiles)
    experts, n, k = weight.shape
    sorted_rows = order.index.shape[0]
    if not (x.is_contiguous() and weight.is_contiguous()) or x.ndim != 2 or x.shape[1] != k or x.dtype != weight.dtype or \
            x.shape[0] != (order.places.shape[0] if gather else sorted_rows):
        raise ValueError("grouped_linear needs contiguous rows and weights [experts, n, k] of one dtype")
    output = torch.empty((sorted_rows, n // 2 if swiglu else n), dtype=x.dtype, device=device)
    rt = runtime(device)
    code = _lib.load().b200_grouped_linear(
        x.data_ptr(), weight.data_ptr(), order.tiles.data_ptr(), order.index.data_ptr() if gather else None,
        order.scores.data_ptr() if swiglu else None, output.data_ptr(), experts, order.tile, order.tiles.shape[0],
        x.shape[0], k, n, _lib.EPILOGUE_SWIGLU if swiglu else _lib.EPILOGUE_NONE, _code(x.dtype),
        rt.status.data_ptr(), _stream())
    _check(code, "b200_grouped_linear")
    _count(rt)
    return output


def sequence_positions(lengths: torch.Tensor, slots: torch.Tensor, positions: torch.Tensor) -> None:
    """positions[r] = lengths[slots[r]], 0 for an idle row."""

    device = _require_cuda(lengths, slots, positions)
    rt = runtime(device)
    _check(_lib.load().b200_sequence_positions(lengths.data_ptr(), slots.data_ptr(), positions.data_ptr(),
                                               slots.shape[0], _stream()), "b200_sequence_positions")
    _count(rt)


def advance_slots(lengths: torch.Tensor, batch: SequenceBatch, capacity: int) -> None:
    """lengths[slot] += the step's tokens of that slot, clamped at `capacity` with a status bit."""

    device = _require_cuda(lengths)
    rt = runtime(device)
    _check(_lib.load().b200_advance_slots(lengths.data_ptr(), batch.slots.data_ptr(), batch.starts.data_ptr(),
                                          batch.sequences, capacity, rt.status.data_ptr(), _stream()),
           "b200_advance_slots")
    _count(rt)
