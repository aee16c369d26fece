"""Vumipel: a decoder whose layers are latent attention or matrix-memory recurrences, normed before and after every
sublayer, with a stretch of layers that runs several times over the same weights.

Configuration and tensors are the checkpoint's; every pass of a looped layer keeps a cache or state of its own."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from . import _lib
from .dense import DTYPES, Arena, DenseLinear, StepInputs, greedy, seq_embed, seq_norm
from .layers import GpuWeights, _dev_index
from .mixers import ClampedGlu, LatentAttention, MatrixMemory, StepContext
from .registry import read_config
from .sequences import OutOfCache, SequenceTable
from .weights import CheckpointWeights

MIXERS = {"latent_attention": LatentAttention, "mlstm": MatrixMemory}


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class VumipelConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[dict, ...]
    loop: Optional[LoopConfig]

    @classmethod
    def from_dict(cls, d: dict) -> "VumipelConfig":
        loop = d.get("loop")
        layers = tuple(d["layers"])
        for i, spec in enumerate(layers):
            if spec["type"] not in MIXERS:
                raise ValueError(f"layer {i}: mixer {spec['type']!r} is not one of {sorted(MIXERS)}")
        if loop is not None:
            loop = LoopConfig(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers, loop)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) in order of execution; the pass is given on the first layer of each pass only."""
        out, i, loop = [], 0, self.loop
        while i < len(self.layers):
            if loop is not None and i == loop.start:
                for t in range(loop.times):
                    out += [(j, t if j == loop.start else None) for j in range(loop.start, loop.stop)]
                i = loop.stop
            else:
                out.append((i, None))
                i += 1
        return out


class VumipelLayer:
    def __init__(self, weights: GpuWeights, i: int, spec: dict, eps: float, dtype: torch.dtype, max_pos: int):
        take = lambda name: weights.take(f"l{i}.{name}").float()
        self.norm1, self.norm1b = take("norm1"), take("norm1b")
        if spec["type"] == "latent_attention":
            self.mixer = LatentAttention(weights, f"l{i}.mix", spec["mixer"], eps, dtype, max_pos)
        else:
            self.mixer = MatrixMemory(weights, f"l{i}.mix", spec["mixer"], eps, dtype)
        self.mlp = None
        if spec.get("mlp") is not None:
            self.norm2, self.norm2b = take("norm2"), take("norm2b")
            self.mlp = ClampedGlu(weights, f"l{i}.mlp", spec["mlp"], dtype)


class HybridState:
    """Device memory of the live sequences: per attention run a paged cache of `num_blocks` blocks (the table's and one spare
    that no sequence owns), per recurrent run a state per slot.  Which blocks and slots belong to whom is the
    `SequenceTable`'s business."""

    def __init__(self, layers, runs, table: SequenceTable, dtype: torch.dtype, device):
        self.spare_block, self.num_blocks = table.num_blocks, table.num_blocks + 1
        self.of_run = []
        for layer, _ in runs:
            m = layers[layer].mixer
            if isinstance(m, LatentAttention):
                self.of_run.append(torch.zeros((self.num_blocks * table.block_size, m.row_size), dtype=dtype, device=device))
            else:
                self.of_run.append(m.state(table.max_sequences, device))

    def nbytes(self) -> int:
        flat = [t for s in self.of_run for t in (s if isinstance(s, tuple) else (s,))]
        return sum(t.numel() * t.element_size() for t in flat)


class Vumipel:
    BLOCK = 64                       # tokens per cache block
    max_portion = 8192               # most tokens of one sequence in a step

    def __init__(self, cfg: VumipelConfig, weights: GpuWeights, device, dtype: str = "bfloat16", max_tokens: int = 8192,
                 max_sequences: int = 8):
        if not torch.cuda.is_available():
            raise _lib.ScratchyCudaError(-5, "Vumipel needs a CUDA device (there is no CPU path)")
        self.cfg, self.device = cfg, torch.device("cuda", _dev_index(device))
        self.dtype = DTYPES[dtype]
        # a sequence may hold all tokens; the others' last blocks are partly filled
        num_blocks = -(-max_tokens // self.BLOCK) + max_sequences
        self.table = SequenceTable(num_blocks, self.BLOCK, max_sequences)
        max_pos = num_blocks * self.BLOCK
        self.embed = weights.take("embed").to(self.dtype).contiguous()
        if tuple(self.embed.shape) != (cfg.vocab, cfg.width):
            raise ValueError(f"`embed` is {tuple(self.embed.shape)}, the configuration says {(cfg.vocab, cfg.width)}")
        self.head = DenseLinear(self.embed)
        self.layers = [VumipelLayer(weights, i, spec, cfg.eps, self.dtype, max_pos) for i, spec in enumerate(cfg.layers)]
        self.final_norm = weights.take("final.norm").float()
        if cfg.loop is not None:
            self.loop_in = DenseLinear(weights.take("loop.in").to(self.dtype))
            self.loop_step = weights.take("loop.step").float().contiguous()
        self.runs = cfg.runs()
        self.state = HybridState(self.layers, self.runs, self.table, self.dtype, self.device)
        self.arena = Arena(self.device)
        self._graphs = {}
        torch.cuda.synchronize(self.device)

    @classmethod
    def from_dir(cls, directory: str, device="cuda", dtype: str = "bfloat16", max_tokens: int = 8192, max_sequences: int = 8) -> "Vumipel":
        device = torch.device("cuda", _dev_index(device))
        return cls(VumipelConfig.from_dict(read_config(directory)), CheckpointWeights.from_dir(directory, device), device, dtype,
                   max_tokens, max_sequences)

    @property
    def vocab(self) -> int:
        return self.cfg.vocab

    # ---- one step
    def _run_step(self, arena: Arena, inputs: StepInputs, entries, logits: Optional[torch.Tensor], max_kv: Optional[int] = None,
                  prompt: bool = False, on_layer=None) -> None:
        """The launches of one step.  `logits`: f32 [wanted, vocab] or None; `on_layer(run, x)`: the residual after every
        layer run (tests)."""
        cfg, T, W, dt = self.cfg, inputs.rows, self.cfg.width, self.dtype
        ctx = StepContext(arena, inputs, inputs.struct(self.table.max_sequences, max_kv), entries, self.table.block_size,
                          self.state.num_blocks, T, prompt)
        x = arena.get("x", (T, W), torch.float32)
        h = arena.get("h", (T, W), dt)
        y = arena.get("y", (T, W), torch.float32)
        cat = arena.get("loop.cat", (T, 2 * W), dt) if cfg.loop is not None else None
        seq_embed(inputs.view("ids"), self.embed, x, None if cat is None else cat[:, W:])
        # `x` is up to date except for `pending` (a sublayer's output and its norm), which joins it in the next norm launch
        pending = {}
        for r, (i, t) in enumerate(self.runs):
            layer = self.layers[i]
            if t is not None:
                seq_norm(x, cfg.eps, out=cat[:, :W], **pending)
                self.loop_in(arena, cat, y)
                pending = {"delta": y, "bias": self.loop_step[t]}
            seq_norm(x, cfg.eps, out=h, w_out=layer.norm1, **pending)
            layer.mixer.run(ctx, h, self.state.of_run[r], y)
            pending = {"delta": y, "w_delta": layer.norm1b}
            if layer.mlp is not None:
                seq_norm(x, cfg.eps, out=h, w_out=layer.norm2, **pending)
                layer.mlp.run(arena, h, y)
                pending = {"delta": y, "w_delta": layer.norm2b}
            if on_layer is not None:
                seq_norm(x, cfg.eps, **pending)
                pending = {}
                on_layer(r, x)
        if logits is None:
            return
        n = int(logits.shape[0])
        hf = arena.get("h.final", (n, W), dt)
        if n == T:                                       # every row, in order
            seq_norm(x, cfg.eps, out=hf, w_out=self.final_norm, **pending)
        else:
            seq_norm(x, cfg.eps, **pending)
            seq_norm(x, cfg.eps, out=hf, w_out=self.final_norm, row_index=inputs.view("want")[:n])
        self.head(arena, hf, logits)

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
            logits = torch.empty((len(rows), self.cfg.vocab), dtype=torch.float32, device=self.device) if rows else None
            prompt = max(n for _, n in counts) >= LatentAttention.EXPAND_FROM
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

    def __init__(self, model: Vumipel, batch: int, max_kv: int):
        dev = model.device
        self.arena = Arena(dev)
        self.inputs = StepInputs(dev, batch, batch, batch, -(-max_kv // model.table.block_size))
        self.logits = torch.empty((batch, model.cfg.vocab), dtype=torch.float32, device=dev)
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
