"""What every sequence model of the package shares: device memory of live sequences, the step's bookkeeping around a
model's own launches, CUDA graphs of decode steps, and greedy sampling.  A design's class states its layers (`_run_step`)."""
from __future__ import annotations

from typing import List, Optional

import torch

from . import _lib
from .dense import DTYPES, Arena, StepInputs, greedy
from .layers import _dev_index
from .mixers import StepContext
from .sequences import OutOfCache, SequenceTable


class HybridState:
    """Device memory of the live sequences: per layer run what its mixer remembers, in a paged cache of `num_blocks` blocks (the
    table's and one spare that no sequence owns) or in state slots.  Which blocks and slots belong to whom is the
    `SequenceTable`'s business."""

    def __init__(self, mixers, table: SequenceTable, device):
        self.spare_block, self.num_blocks = table.num_blocks, table.num_blocks + 1
        self.of_run = [m.memory(self.num_blocks * table.block_size, table.max_sequences, device) for m in mixers]

    def nbytes(self) -> int:
        def size(s) -> int:
            return s.numel() * s.element_size() if isinstance(s, torch.Tensor) else sum(size(t) for t in s)
        return sum(size(s) for s in self.of_run)


class HybridModel:
    """`mixers`: the mixer of every layer run, in order of execution."""
    BLOCK = 64                       # tokens per cache block
    max_portion = 8192               # most tokens of one sequence in a step
    prompt_rows = 64                 # rows of one sequence from which a step counts as a prompt

    def __init__(self, vocab: int, width: int, device, dtype: str, max_tokens: int, max_sequences: int, window: Optional[int] = None,
                 keep_first: int = 0):
        if not torch.cuda.is_available():
            raise _lib.ScratchyCudaError(-5, f"{type(self).__name__} needs a CUDA device (there is no CPU path)")
        self.vocab, self.width = vocab, width
        self.device, self.dtype = torch.device("cuda", _dev_index(device)), DTYPES[dtype]
        # a sequence may hold all tokens; the others' last blocks are partly filled
        num_blocks = -(-max_tokens // self.BLOCK) + max_sequences
        self.table = SequenceTable(num_blocks, self.BLOCK, max_sequences, window, keep_first)
        self.arena = Arena(self.device)
        self._graphs = {}

    def _take_embedding(self, weights) -> torch.Tensor:
        embed = weights.take("embed").to(self.dtype).contiguous()
        if tuple(embed.shape) != (self.vocab, self.width):
            raise ValueError(f"`embed` is {tuple(embed.shape)}, the configuration says {(self.vocab, self.width)}")
        return embed

    def _open_state(self, mixers) -> None:
        self.state = HybridState(mixers, self.table, self.device)
        torch.cuda.synchronize(self.device)

    # ---- one step
    def _run_step(self, arena: Arena, inputs: StepInputs, entries, logits: Optional[torch.Tensor], max_kv: Optional[int] = None,
                  prompt: bool = False, on_layer=None) -> None:
        """The launches of one step.  `logits`: f32 [wanted, vocab] or None; `on_layer(run, x)`: the residual after every
        layer run (tests)."""
        raise NotImplementedError

    def _context(self, arena: Arena, inputs: StepInputs, entries, max_kv: Optional[int], prompt: bool) -> StepContext:
        return StepContext(arena, inputs, inputs.struct(self.table.max_sequences, max_kv), entries, self.table.block_size, self.state.num_blocks,
                           inputs.rows, prompt)

    def forward(self, entries, want, on_layer=None) -> Optional[torch.Tensor]:
        """Runs the tokens of `entries` [(Sequence, token ids)] and returns f32 logits [number wanted, vocab] for the places
        `want[e]` (ascending indices into entry e's tokens), or None when nothing is wanted.  Reserves cache blocks first
        (`OutOfCache` leaves everything as it was)."""
        table = self.table
        if sum(table.blocks_needed(seq, len(tok)) for seq, tok in entries) > table.free_blocks:
            raise OutOfCache("not enough free cache blocks for this step")
        rows, base = [], 0
        for (seq, tok), places in zip(entries, want):
            if not tok:
                raise ValueError("an entry without tokens")
            if any(not 0 <= p < len(tok) for p in places):
                raise ValueError("a wanted place outside the entry's tokens")
            rows += [base + p for p in places]
            base += len(tok)
        for seq, tok in entries:
            table.extend(seq, len(tok))
        counts = [(seq, len(tok)) for seq, tok in entries]
        if on_layer is None and base == len(entries) and rows == list(range(base)) and base <= 64:
            logits = self._decode(entries)
        else:
            inputs = StepInputs(self.device, base, len(entries), len(rows), max(len(seq.blocks) for seq, _ in entries))
            inputs.fill(entries, rows)
            # logits of every row in order skip the gather; any other selection goes through the row index
            logits = torch.empty((len(rows), self.vocab), dtype=torch.float32, device=self.device) if rows else None
            prompt = max(n for _, n in counts) >= self.prompt_rows
            self._run_step(self.arena, inputs, counts, logits, prompt=prompt, on_layer=on_layer)
            torch.cuda.current_stream(self.device).synchronize()         # `inputs` may be dropped now
        for seq, n in counts:
            table.advance(seq, n)
        return logits

    # ---- decoding: one token per sequence, the whole step one CUDA graph
    def _decode(self, entries) -> torch.Tensor:
        batch = len(entries)
        kv = max(seq.length + 1 for seq, _ in entries)
        bucket = self.table.block_size * 4
        while bucket < kv:
            bucket *= 2
        g = self.decode_graph(batch, bucket)
        g.inputs.fill(entries, list(range(batch)))
        g.graph.replay()
        torch.cuda.current_stream(self.device).synchronize()
        return g.logits.clone()

    def decode_graph(self, batch: int, max_kv: int) -> "DecodeGraph":
        """The captured decode step of `batch` sequences with up to `max_kv` tokens each (captured on first use)."""
        key = (batch, max_kv)
        if key not in self._graphs:
            self._graphs[key] = DecodeGraph(self, batch, max_kv)
        return self._graphs[key]

    def check_health(self) -> None:
        """Raises if a device-side check fired since the last call (`scr_device_status`)."""
        _lib.models_context(_dev_index(self.device)).device_status(None)

    def greedy(self, logits: torch.Tensor) -> List[int]:
        return greedy(logits).tolist()


class DecodeGraph:
    """A decode step with buffers of its own, captured once and replayed."""

    def __init__(self, model: HybridModel, batch: int, max_kv: int):
        dev = model.device
        self.arena = Arena(dev)
        self.inputs = StepInputs(dev, batch, batch, batch, -(-max_kv // model.table.block_size))
        self.logits = torch.empty((batch, model.vocab), dtype=torch.float32, device=dev)
        self.next_ids = torch.zeros(batch, dtype=torch.int32, device=dev)
        # the warm-up step sizes the buffers: its segments are empty (no state is touched) and its cache rows land in the
        # spare block that no sequence owns
        self.inputs.max_count, self.inputs.max_kv = 1, max_kv
        self.inputs.view("table").fill_(model.state.spare_block)
        stream = torch.cuda.Stream(dev)
        stream.wait_stream(torch.cuda.current_stream(dev))

        def step():
            model._run_step(self.arena, self.inputs, [], self.logits, max_kv=max_kv)
            greedy(self.logits, self.next_ids)
        with torch.cuda.stream(stream):
            step()
        torch.cuda.current_stream(dev).wait_stream(stream)
        torch.cuda.synchronize(dev)
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph, stream=stream):
            step()
