"""Vekurax: a decoder whose layers add three branches of one normed input to the residual: sliding-window attention,
lightning attention and a feed-forward.  Its norms are dynamic tanh.  A layer may run again further up on the weights of an
earlier one, with a cache and a state of its own."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .dense import Arena, DenseLinear, StepInputs, TanhNorm, seq_embed, seq_norm
from .hybrid import HybridModel
from .layers import GpuWeights, _dev_index
from .mixers import GeluGlu, LightningAttention, SideBySide, WindowAttention
from .registry import read_config
from .weights import CheckpointWeights


@dataclass(frozen=True)
class VekuraxConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[dict, ...]

    @classmethod
    def from_dict(cls, d: dict) -> "VekuraxConfig":
        layers = tuple(d["layers"])
        for i, spec in enumerate(layers):
            if spec["type"] != "parallel":
                raise ValueError(f"layer {i}: mixer {spec['type']!r} is not 'parallel'")
            j = spec.get("weights_of")
            if j is not None and not 0 <= j < i:
                raise ValueError(f"layer {i} can not use the weights of layer {j}")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers)

    def owners(self) -> List[int]:
        """For every layer the one whose tensors it runs on."""
        out = []
        for i, spec in enumerate(self.layers):
            j = spec.get("weights_of")
            out.append(i if j is None else out[j])
        return out

    @property
    def window(self) -> int:
        return max(int(s["mixer"]["left"]["mask"]["size"]) for s in self.layers)

    @property
    def keep_first(self) -> int:
        return max(int(s["mixer"]["left"]["mask"]["keep_first"]) for s in self.layers)


class VekuraxLayer:
    def __init__(self, weights: GpuWeights, i: int, spec: dict, eps: float, dtype: torch.dtype):
        m = spec["mixer"]
        self.norm1 = TanhNorm.take(weights, f"l{i}.norm1")
        mlp = None if spec.get("mlp") is None else GeluGlu(weights, f"l{i}.mlp", spec["mlp"], dtype)
        self.branches = SideBySide([WindowAttention(weights, f"l{i}.mix.left", m["left"], eps, dtype, float(m["left_scale"])),
                                    LightningAttention(weights, f"l{i}.mix.right", m["right"], eps, dtype, float(m["right_scale"]))], mlp)


class Vekurax(HybridModel):
    def __init__(self, cfg: VekuraxConfig, weights: GpuWeights, device, dtype: str = "bfloat16", max_tokens: int = 8192,
                 max_sequences: int = 8):
        super().__init__(cfg.vocab, cfg.width, device, dtype, max_tokens, max_sequences, cfg.window, cfg.keep_first)
        self.cfg = cfg
        self.embed = self._take_embedding(weights)
        self.head = DenseLinear(self.embed)
        layers = {i: VekuraxLayer(weights, i, cfg.layers[i], cfg.eps, self.dtype) for i in sorted(set(cfg.owners()))}
        self.layers = [layers[i] for i in cfg.owners()]                              # in order of execution
        self.final_norm = TanhNorm.take(weights, "final.norm")
        self._open_state([layer.branches for layer in self.layers])

    @classmethod
    def from_dir(cls, directory: str, device="cuda", dtype: str = "bfloat16", max_tokens: int = 8192, max_sequences: int = 8) -> "Vekurax":
        device = torch.device("cuda", _dev_index(device))
        return cls(VekuraxConfig.from_dict(read_config(directory)), CheckpointWeights.from_dir(directory, device), device, dtype,
                   max_tokens, max_sequences)

    def _run_step(self, arena: Arena, inputs: StepInputs, entries, logits: Optional[torch.Tensor], max_kv: Optional[int] = None,
                  prompt: bool = False, on_layer=None) -> None:
        cfg, T, W = self.cfg, inputs.rows, self.cfg.width
        ctx = self._context(arena, inputs, entries, max_kv, prompt)
        x = arena.get("x", (T, W), torch.float32)
        h = arena.get("h", (T, W), self.dtype)
        seq_embed(inputs.view("ids"), self.embed, x)
        seq_norm(x, cfg.eps, out=h, tanh=self.layers[0].norm1)
        every = logits is not None and int(logits.shape[0]) == T
        for r, layer in enumerate(self.layers):
            # the layer's last launch leaves the norm that comes next; few wanted rows are normed on their own
            last = r + 1 == len(self.layers)
            norm = self.layers[r + 1].norm1 if not last else self.final_norm if every else None
            layer.branches.run(ctx, h, self.state.of_run[r], x, norm)
            if on_layer is not None:
                on_layer(r, x)
        if logits is None:
            return
        if not every:
            n = int(logits.shape[0])
            h = arena.get("h.final", (n, W), self.dtype)
            seq_norm(x, cfg.eps, out=h, tanh=self.final_norm, row_index=inputs.view("want")[:n])
        self.head(arena, h, logits)
