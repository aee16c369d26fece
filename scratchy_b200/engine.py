"""The serving engine: steps over live sequences, a scheduler that admits requests and batches their tokens, and greedy
sampling.  Models come from the registry and are driven through one interface (registry.py), so a replayed trace, a
generation and a benchmark run the same step."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Deque, Dict, Hashable, List, Optional, Sequence as Seq, Tuple

import torch

from .sequences import OutOfCache, Sequence


@dataclass
class Request:
    """A prompt and what has been generated for it."""
    name: Hashable
    prompt: List[int]
    max_new_tokens: int
    stop_ids: Tuple[int, ...] = ()
    output: List[int] = field(default_factory=list)
    done: bool = False


class Engine:
    """`step_tokens`: most prompt tokens a step takes.  A step is either portions of prompts or one token of every sequence
    that is decoding (each kind has kernels of its own); prompts come first, so that waiting requests join the batch soon."""

    def __init__(self, model, step_tokens: int = 2048, max_batch: int = 32):
        self.model, self.table = model, model.table
        self.step_tokens = max(1, step_tokens)
        self.max_batch = max(1, min(max_batch, self.table.max_sequences))
        self.waiting: Deque[Request] = deque()
        self.running: Dict[Hashable, Request] = {}
        self._serial = 0

    # ---- the step, for callers that bring their own tokens
    def run_step(self, entries: Seq[Tuple[Hashable, List[int], List[int]]], end: Seq[Hashable] = ()) -> Optional[torch.Tensor]:
        """`entries`: (sequence name, its next tokens, wanted places among them).  Unknown names open a sequence; `end` closes
        sequences after the step.  Returns f32 logits of the wanted places in order, or None."""
        table, pieces = self.table, []
        live = [(table.live[name] if name in table.live else table.open(name), list(tokens), sorted_places(places))
                for name, tokens, places in entries if tokens]
        limit = self.model.max_portion
        at = [0] * len(live)
        while any(at[e] < len(tokens) for e, (_, tokens, _) in enumerate(live)):
            part, want, who = [], [], []
            for e, (seq, tokens, places) in enumerate(live):
                lo, hi = at[e], min(at[e] + limit, len(tokens))
                if lo == hi:
                    continue
                part.append((seq, tokens[lo:hi]))
                want.append([p - lo for p in places if lo <= p < hi])
                who.append(e)
                at[e] = hi
            logits = self.model.forward(part, want)
            row = 0
            for e, places in zip(who, want):
                if places:
                    pieces.append((e, logits[row:row + len(places)]))
                row += len(places)
        for name in end:
            if name in table.live:
                table.close(name)
        pieces.sort(key=lambda p: p[0])
        return torch.cat([p for _, p in pieces]) if pieces else None

    # ---- the scheduler
    def submit(self, prompt: Seq[int], max_new_tokens: int, stop_ids: Seq[int] = (), name: Hashable = None) -> Request:
        if not prompt or max_new_tokens < 1:
            raise ValueError("a request needs a prompt and at least one token to generate")
        if any(not 0 <= t < self.model.vocab for t in prompt):
            raise ValueError("token id outside the vocabulary")
        longest = len(prompt) + max_new_tokens
        if self.table.most_blocks(longest, self._portion) > self.table.num_blocks:
            raise ValueError(f"{longest} tokens do not fit a cache of {self.table.num_blocks * self.table.block_size}")
        self._serial += 1
        req = Request(name if name is not None else ("request", self._serial), list(prompt), max_new_tokens, tuple(stop_ids))
        self.waiting.append(req)
        return req

    @property
    def _portion(self) -> int:
        return min(self.step_tokens, self.model.max_portion)

    def _blocks_to_finish(self, req: Request, seq: Optional[Sequence]) -> int:
        have = seq.held if seq is not None else 0
        return max(0, self.table.most_blocks(len(req.prompt) + req.max_new_tokens, self._portion) - have)

    def _admit(self) -> None:
        """Waiting requests in order, each only if everything that runs can still finish: a running sequence never has to be
        thrown out."""
        reserved = sum(self._blocks_to_finish(r, self.table.live[n]) for n, r in self.running.items())
        while self.waiting and len(self.running) < self.max_batch and self.table.free_slots:
            need = self._blocks_to_finish(self.waiting[0], None)
            if reserved + need > self.table.free_blocks:
                break
            req = self.waiting.popleft()
            self.table.open(req.name)
            self.running[req.name] = req
            reserved += need

    def _plan(self) -> List[Tuple[Request, Sequence, List[int], bool]]:
        """(request, sequence, tokens, does the last token's logits matter)."""
        plan, budget = [], self.step_tokens
        for name, req in self.running.items():
            seq = self.table.live[name]
            left = len(req.prompt) - seq.length
            if left > 0 and budget > 0:
                n = min(left, budget, self.model.max_portion)
                plan.append((req, seq, req.prompt[seq.length:seq.length + n], n == left))
                budget -= n
        if plan:
            return plan
        return [(req, self.table.live[name], [req.output[-1]], True) for name, req in self.running.items()]

    def schedule_step(self) -> bool:
        """Admit, run one step, sample.  False when nothing is left to do."""
        self._admit()
        if not self.running:
            if self.waiting:
                raise OutOfCache("a waiting request can not be admitted although nothing runs")
            return False
        plan = self._plan()
        logits = self.model.forward([(seq, tokens) for _, seq, tokens, _ in plan], [[len(t) - 1] if last else [] for _, _, t, last in plan])
        sampled = self.model.greedy(logits) if logits is not None else []
        for (req, seq, _, last) in plan:
            if not last:
                continue
            token = sampled.pop(0)
            req.output.append(token)
            if len(req.output) >= req.max_new_tokens or token in req.stop_ids:
                req.done = True
                self.table.close(req.name)
                del self.running[req.name]
        return True

    def generate(self, prompts: Seq[Seq[int]], max_new_tokens: int, stop_ids: Seq[int] = ()) -> List[List[int]]:
        """Greedy continuations of the prompts, in their order."""
        reqs = [self.submit(p, max_new_tokens, stop_ids) for p in prompts]
        while self.schedule_step():
            pass
        self.model.check_health()
        return [r.output for r in reqs]


def sorted_places(places: Seq[int]) -> List[int]:
    out = list(places)
    if out != sorted(set(out)):
        raise ValueError("wanted places must be ascending and distinct")
    return out
