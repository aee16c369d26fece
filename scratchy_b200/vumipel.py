"""Vumipel: a decoder whose layers are latent attention or matrix-memory recurrences, normed before and after every
sublayer, with a stretch of layers that runs several times over the same weights.

Configuration and tensors are the checkpoint's; every pass of a looped layer keeps a cache or state of its own."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .dense import Arena, DenseLinear, StepInputs, seq_embed, seq_norm
from .hybrid import HybridModel
from .layers import GpuWeights, _dev_index
from .mixers import ClampedGlu, LatentAttention, MatrixMemory
from .registry import read_config
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


class Vumipel(HybridModel):
    def __init__(self, cfg: VumipelConfig, weights: GpuWeights, device, dtype: str = "bfloat16", max_tokens: int = 8192,
                 max_sequences: int = 8):
        super().__init__(cfg.vocab, cfg.width, device, dtype, max_tokens, max_sequences)
        self.cfg = cfg
        max_pos = self.table.num_blocks * self.BLOCK
        self.embed = self._take_embedding(weights)
        self.head = DenseLinear(self.embed)
        self.layers = [VumipelLayer(weights, i, spec, cfg.eps, self.dtype, max_pos) for i, spec in enumerate(cfg.layers)]
        self.final_norm = weights.take("final.norm").float()
        if cfg.loop is not None:
            self.loop_in = DenseLinear(weights.take("loop.in").to(self.dtype))
            self.loop_step = weights.take("loop.step").float().contiguous()
        self.runs = cfg.runs()
        self._open_state([self.layers[i].mixer for i, _ in self.runs])

    @classmethod
    def from_dir(cls, directory: str, device="cuda", dtype: str = "bfloat16", max_tokens: int = 8192, max_sequences: int = 8) -> "Vumipel":
        device = torch.device("cuda", _dev_index(device))
        return cls(VumipelConfig.from_dict(read_config(directory)), CheckpointWeights.from_dir(directory, device), device, dtype,
                   max_tokens, max_sequences)

    def _run_step(self, arena: Arena, inputs: StepInputs, entries, logits: Optional[torch.Tensor], max_kv: Optional[int] = None,
                  prompt: bool = False, on_layer=None) -> None:
        cfg, T, W, dt = self.cfg, inputs.rows, self.cfg.width, self.dtype
        ctx = self._context(arena, inputs, entries, max_kv, prompt)
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
