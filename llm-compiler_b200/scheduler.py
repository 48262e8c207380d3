"""Continuous batching over an engine's step function: requests arrive at any time, prompts are run in
portions of a bounded number of tokens, and all running sequences decode together.

The engine provides open() / close(slot), forward(entries), decode_rows(slots, tokens), batch (slots)
and capacity (tokens a slot holds). Sampling is greedy (the engine's argmax kernel)."""

from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Deque, List, Optional, Sequence

from . import kernels
from .kv_state import ExecutionError


@dataclass
class Request:
    prompt: List[int]
    max_new_tokens: int
    stop_token: Optional[int] = None
    output: List[int] = field(default_factory=list)
    slot: Optional[int] = None
    done_tokens: int = 0  # tokens of the prompt that have been run
    finished: bool = False


class RequestScheduler:
    def __init__(self, engine, *, max_portion: int = 2048, use_graphs: bool = True) -> None:
        if max_portion <= 0:
            raise ValueError("a portion holds at least one token")
        self.engine = engine
        self.max_portion = max_portion  # prompt tokens run between two decode steps
        self.use_graphs = use_graphs
        self.waiting: Deque[Request] = deque()
        self.prompting: List[Request] = []
        self.running: List[Request] = []

    def submit(self, prompt: Sequence[int], max_new_tokens: int, *, stop_token: Optional[int] = None) -> Request:
        if not prompt or max_new_tokens <= 0:
            raise ValueError("a request needs a prompt and at least one new token")
        if len(prompt) + max_new_tokens - 1 > self.engine.capacity:
            raise ExecutionError(f"a request of {len(prompt)} + {max_new_tokens} tokens exceeds the slot capacity "
                                 f"{self.engine.capacity}")
        request = Request([int(t) for t in prompt], int(max_new_tokens), stop_token)
        self.waiting.append(request)
        return request

    @property
    def idle(self) -> bool:
        return not (self.waiting or self.prompting or self.running)

    def _admit(self) -> None:
        while self.waiting and len(self.prompting) + len(self.running) < self.engine.batch:
            request = self.waiting.popleft()
            request.slot = self.engine.open()
            self.prompting.append(request)

    def _take(self, request: Request, token: int) -> bool:
        request.output.append(token)
        if len(request.output) >= request.max_new_tokens or token == request.stop_token:
            request.finished = True
            self.engine.close(request.slot)
            request.slot = None
        return request.finished

    def step(self) -> List[Request]:
        """Admits what fits, runs at most `max_portion` prompt tokens, then one decode step of every
        running sequence. Returns the requests that finished."""

        self._admit()
        finished: List[Request] = []
        decoding = list(self.running)
        budget = self.max_portion
        entries, portions = [], []
        for request in self.prompting:
            if budget == 0:
                break
            count = min(budget, len(request.prompt) - request.done_tokens)
            entries.append((request.slot, request.prompt[request.done_tokens:request.done_tokens + count]))
            portions.append((request, count))
            budget -= count
        if entries:
            ends = [r.done_tokens + count == len(r.prompt) for r, count in portions]
            logits = self.engine.forward(entries, [[len(tokens) - 1] if end else []
                                                   for (_, tokens), end in zip(entries, ends)])
            first = kernels.b200_argmax(logits).tolist() if logits is not None else []
            for (request, count), end in zip(portions, ends):
                request.done_tokens += count
                if end:
                    self.prompting.remove(request)
                    if self._take(request, first.pop(0)):
                        finished.append(request)
                    else:
                        self.running.append(request)
        if decoding:
            tokens = self.engine.decode_rows([r.slot for r in decoding], [r.output[-1] for r in decoding],
                                             use_graph=self.use_graphs)
            for request, token in zip(decoding, tokens):
                if self._take(request, token):
                    self.running.remove(request)
                    finished.append(request)
        self.engine.state.check()
        return finished

    def run(self) -> None:
        while not self.idle:
            self.step()
