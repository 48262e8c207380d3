"""Serving engine of the hybrid designs: layers whose mixers keep recurrent state, cached latents or
keys and values in slots, an fp32 residual stream, portions of prompts and decoded tokens through one step function.

`forward` is the step: it takes, for any number of sequences, the next tokens of each (a whole prompt, a
portion of one, or one decoded token) and runs them from the state that earlier steps left. `prefill`,
`decode_step`, `step` and `generate` are the fixed-batch interface of every engine here (ReplicaServer
serves either); `decode_rows` is the batched decode step of the request scheduler, replayed from a CUDA
graph per batch size."""

from __future__ import annotations

import os
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from . import hybrid_kernels as hk
from . import kernels
from .engine import ServingEngine
from .hybrid_kernels import SequenceBatch, pad8
from .kv_state import ExecutionError, SlotState
from .mixers import pad_matrix


class HybridEngine(ServingEngine):
    def __init__(self, config, weights: Dict[str, torch.Tensor], *, batch: int,
                 capacity: int, device: Optional[torch.device] = None) -> None:
        """`batch` slots of `capacity` tokens each. `config`: a hybrid design's (bazirax, lozanex): sizes,
        norm_eps, norm_offset and build_layers(weights). The weights' dtype (fp32 or bf16) is the dtype of
        projections and caches; they must be on the device."""

        for name, tensor in weights.items():
            if not tensor.is_cuda:
                raise ValueError(f"weight {name} is not on a CUDA device")
        self._init_step(batch, device or torch.device("cuda", torch.cuda.current_device()))
        self.config = config
        self.capacity = capacity
        self.dtype = weights["embed"].dtype
        self.epsilon, self.norm_offset = config.norm_eps, config.norm_offset
        self.layers = config.build_layers(weights)
        self.embed, self.embed_norm = weights["embed"], weights.get("embed.norm")
        self.final_norm = weights["final.norm"]
        self.head = pad_matrix(weights["head"], pad8(config.vocab_size), pad8(config.hidden_size))
        self.state = SlotState([layer.mixer.state_spec(capacity) for layer in self.layers], slots=batch,
                               capacity=capacity, device=self.device)
        int32 = dict(dtype=torch.int32, device=self.device)
        # the vectors of a decode step, at fixed addresses: row r decodes for slot row_slots[r]
        self.row_slots = torch.arange(batch, **int32)
        self._row_bases = torch.zeros(batch, **int32)
        self._row_starts = torch.arange(batch + 1, **int32)
        self._row_sequence = torch.arange(batch, **int32)
        self._host_slots = torch.zeros(batch, dtype=torch.int32).pin_memory()
        self.programmatic_launch = os.environ.get("B200_PROGRAMMATIC_LAUNCH", "1") != "0"
        self._row_graphs: Dict[int, Tuple[torch.cuda.CUDAGraph, torch.Tensor]] = {}

    # ------------------------------------------------------------------ the layers ----
    def _norm_step(self, x, y, post_weight, next_weight, narrow=False):
        return hk.residual_norm(x, y, post_weight, next_weight, epsilon=self.epsilon,
                                weight_offset=self.norm_offset, dtype=self.dtype, narrow=narrow)

    def _run_layers(self, ids: torch.Tensor, batch: SequenceBatch, last_norm: Optional[torch.Tensor],
                    streams: Optional[list] = None) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """Residual stream behind the last layer, and its rows normed with `last_norm`."""

        first = self.layers[0].norm_in
        x = hk.embedding_residual(self.embed, ids, self.embed_norm, epsilon=self.epsilon,
                                  weight_offset=self.norm_offset, narrow=first is None)
        if first is None:
            x, h = x
        else:
            h = self._norm_step(x, None, None, first)
        for index, layer in enumerate(self.layers):
            last = index + 1 == len(self.layers)
            after = last_norm if last else self.layers[index + 1].norm_in
            source = layer.mixer.shared_state
            y = layer.mixer(h, batch, self.state.layers[index if source is None else source])
            if layer.mlp is not None:
                h = self._norm_step(x, y, layer.norm_out, layer.mlp_norm_in, narrow=layer.mlp_norm_in is None)
                h = self._norm_step(x, layer.mlp(h), layer.mlp_norm_out, after, narrow=not last and after is None)
            else:
                h = self._norm_step(x, y, layer.norm_out, after, narrow=not last and after is None)
            if streams is not None:
                streams.append(x.clone())
        return x, h

    def _logits(self, h: torch.Tensor) -> torch.Tensor:
        return kernels.b200_linear(h, self.head)[:, :self.config.vocab_size]

    # -------------------------------------------------------------------- the step ----
    def open(self) -> int:
        """A slot for a new sequence."""

        return self.state.acquire()

    def close(self, slot: int) -> None:
        self.state.release(slot)

    def forward(self, entries: Sequence[Tuple[int, Sequence[int]]],
                want: Optional[Sequence[Sequence[int]]] = None, *,
                streams: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the next tokens of each entry (slot, tokens). `want[i]`: the places among entry i's
        tokens whose logits are asked for (default: each entry's last). Returns the logits of the
        wanted places in order, [wanted, vocab] in the model dtype, or None if there are none."""

        slots = [slot for slot, _ in entries]
        counts = [len(tokens) for _, tokens in entries]
        ids = torch.tensor([t for _, tokens in entries for t in tokens], dtype=torch.int64)
        return self._forward_ids(ids, slots, counts, want, streams)

    def _forward_ids(self, ids: torch.Tensor, slots: List[int], counts: List[int],
                     want: Optional[Sequence[Sequence[int]]], streams: Optional[list] = None) -> Optional[torch.Tensor]:
        if not slots or min(counts) == 0 or len(set(slots)) != len(slots):
            raise ValueError("every entry needs a slot of its own and at least one token")
        for slot, count in zip(slots, counts):
            self.state.require(slot, count)
        bases = [self.state.host_lengths[slot] for slot in slots]
        starts = [0]
        for count in counts:
            starts.append(starts[-1] + count)
        rows, n = starts[-1], len(slots)
        if want is None:
            want = [[count - 1] for count in counts]
        if any(not 0 <= place < counts[i] for i, places in enumerate(want) for place in places):
            raise ValueError("a wanted place lies outside its entry")
        wanted = [starts[i] + place for i, places in enumerate(want) for place in places]
        ids = ids.to(self.device)
        packed = torch.cat([torch.repeat_interleave(torch.arange(n, dtype=torch.int32), torch.tensor(counts)),
                            torch.tensor(starts + slots + bases, dtype=torch.int32)]).to(self.device)
        batch = SequenceBatch(rows, n, packed[:rows], packed[rows:rows + n + 1],
                              packed[rows + n + 1:rows + 2 * n + 1], packed[rows + 2 * n + 1:], counts, bases, slots)
        x, _ = self._run_layers(ids, batch, None, streams)
        hk.advance_slots(self.state.lengths, batch, self.capacity)
        for slot, count in zip(slots, counts):
            self.state.host_lengths[slot] += count
        if not wanted:
            return None
        if wanted != list(range(rows)):
            x = kernels.b200_embedding(x, torch.tensor(wanted, dtype=torch.int64).to(self.device))
        return self._logits(self._norm_step(x, None, None, self.final_norm))

    # ---------------------------------------------------------------------- decode ----
    def _decode_rows(self, rows: int) -> torch.Tensor:
        """One token for each of the first `rows` rows of the step's vectors; returns the logits."""

        before = kernels.launch_count(self.device)
        batch = SequenceBatch(rows, rows, self._row_sequence[:rows], self._row_starts[:rows + 1],
                              self.row_slots[:rows], self._row_bases[:rows])
        # The step opens with fully serialised launches (positions, embedding), weights are written once,
        # and a layer's recurrent state by that layer's own step kernel only: the kernels behind may
        # fetch weights and state before their predecessor has finished.
        with kernels.launch_mode(programmatic=self.programmatic_launch, constant_weights=self.programmatic_launch,
                                 stable_kv_prefix=self.programmatic_launch):
            hk.sequence_positions(self.state.lengths, batch.slots, batch.bases)
            _, h = self._run_layers(self.input_ids[:rows], batch, self.final_norm)
            logits = self._logits(h)
        kernels.b200_argmax(logits, self.next_ids[:rows])
        hk.advance_slots(self.state.lengths, batch, self.capacity)
        self.kernels_per_step = kernels.launch_count(self.device) - before
        return logits

    def _decode_step(self) -> None:
        self.logits = self._decode_rows(self.batch)

    def _warm_up(self) -> None:
        saved = self.row_slots.clone()
        self.row_slots.fill_(-1)  # idle rows leave no trace
        self._decode_rows(self.batch)
        self.row_slots.copy_(saved)

    def _count_step(self) -> None:
        for slot in range(self.batch):
            self.state.host_lengths[slot] += 1

    def prefill(self, input_ids: torch.Tensor) -> torch.Tensor:
        """A B x T prompt from empty state, one sequence per slot; returns the last positions' logits
        and primes the greedy next token."""

        if input_ids.ndim != 2 or input_ids.shape[0] != self.batch:
            raise ValueError("prompt must be batch x tokens")
        self.state.reset_all()
        self.row_slots.copy_(torch.arange(self.batch, dtype=torch.int32))
        self.logits = self._forward_ids(input_ids.reshape(-1), list(range(self.batch)),
                                        [input_ids.shape[1]] * self.batch, None)
        kernels.b200_argmax(self.logits, self.next_ids)
        self.input_ids.copy_(self.next_ids)
        return self.logits

    def load_context(self, lengths: Sequence[int]) -> None:
        """Benchmark entry: declares that slot b holds a context of lengths[b] tokens, whatever its
        state tensors contain."""

        self.state.reset_all()
        self.state.host_lengths = [int(n) for n in lengths]
        self.state.lengths.copy_(torch.tensor(self.state.host_lengths, dtype=torch.int64))
        self.row_slots.copy_(torch.arange(self.batch, dtype=torch.int32))

    def decode_rows(self, slots: Sequence[int], tokens: Sequence[int], *, use_graph: bool = True) -> List[int]:
        """One decode step of the sequences in `slots`, fed with `tokens`: their greedy next tokens.
        Batches are rounded up to a power of two with idle rows, one captured graph for each."""

        count = len(slots)
        if count == 0 or count > self.batch or len(set(slots)) != count:
            raise ValueError("a decode step takes one row per slot")
        for slot in slots:
            self.state.require(slot, 1)
        rows = 1
        while rows < count:
            rows *= 2
        rows = min(rows, self.batch)
        self._host_slots[:rows] = torch.tensor(list(slots) + [-1] * (rows - count), dtype=torch.int32)
        self._host_ids[:rows] = torch.tensor(list(tokens) + [0] * (rows - count), dtype=torch.int64)
        if use_graph and rows not in self._row_graphs:
            self._capture_rows(rows)
        self.row_slots[:rows].copy_(self._host_slots[:rows], non_blocking=True)
        self.input_ids[:rows].copy_(self._host_ids[:rows], non_blocking=True)
        if use_graph:
            graph, logits = self._row_graphs[rows]
            graph.replay()
        else:
            logits = self._decode_rows(rows)
        self.logits = logits[:count]
        self._host_tokens[:rows].copy_(self.next_ids[:rows], non_blocking=True)
        for slot in slots:
            self.state.host_lengths[slot] += 1
        torch.cuda.current_stream(self.device).synchronize()
        return self._host_tokens[:count].tolist()

    def _capture_rows(self, rows: int) -> None:
        saved = self.row_slots.clone()
        self.row_slots.fill_(-1)
        stream = torch.cuda.Stream(device=self.device)
        stream.wait_stream(torch.cuda.current_stream(self.device))
        with torch.cuda.stream(stream):
            self._decode_rows(rows)
        torch.cuda.current_stream(self.device).wait_stream(stream)
        torch.cuda.synchronize(self.device)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            logits = self._decode_rows(rows)
        self._row_graphs[rows] = (graph, logits)
        self.row_slots.copy_(saved)
