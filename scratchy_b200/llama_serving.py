"""The int4 Llama decoder behind the serving interface of the registry: checkpoint folder in, steps of one token per
sequence (a prompt runs token by token through the decode step), block and slot bookkeeping by a `SequenceTable`."""
from __future__ import annotations

from typing import List, Optional

import torch

from . import _lib
from .decode import DecodeBuffers, LlamaConfig, LlamaDecoder, PagedKvCache, argmax
from .layers import _dev_index
from .registry import read_config
from .sequences import OutOfCache, SequenceTable
from .weights import CheckpointWeights


def config_from_dict(d: dict) -> LlamaConfig:
    heads = int(d["num_attention_heads"])
    quant = d.get("quantization") or d.get("quantization_config") or {}
    return LlamaConfig(hidden=int(d["hidden_size"]), n_layers=int(d["num_hidden_layers"]), n_q_heads=heads,
                       n_kv_heads=int(d.get("num_key_value_heads", heads)), head_dim=int(d.get("head_dim", int(d["hidden_size"]) // heads)),
                       intermediate=int(d["intermediate_size"]), vocab=int(d["vocab_size"]), rms_eps=float(d.get("rms_norm_eps", 1e-5)),
                       rope_theta=float(d.get("rope_theta", 500000.0)), group_size=int(quant.get("group_size", 64)))


class LlamaServing:
    BLOCK = 16
    max_portion = 1

    def __init__(self, cfg: LlamaConfig, checkpoint, device, max_tokens: int = 8192, max_sequences: int = 8):
        self.device = torch.device("cuda", _dev_index(device))
        num_blocks = -(-max_tokens // self.BLOCK) + max_sequences
        self.table = SequenceTable(num_blocks, self.BLOCK, max_sequences)
        self.decoder = LlamaDecoder(cfg, checkpoint, self.device, max_pos=num_blocks * self.BLOCK)
        self.cache = PagedKvCache(cfg, num_blocks, self.BLOCK, self.device)
        self.vocab = cfg.vocab
        self._buffers = {}

    @classmethod
    def from_dir(cls, directory: str, device="cuda", dtype: str = "bfloat16", max_tokens: int = 8192, max_sequences: int = 8) -> "LlamaServing":
        if dtype != "bfloat16":
            raise _lib.ScratchyCudaError(-4, f"the int4 Llama decoder runs in bfloat16, not {dtype}")
        return cls(config_from_dict(read_config(directory)), CheckpointWeights.from_dir(directory, torch.device("cuda", _dev_index(device))),
                   device, max_tokens, max_sequences)

    def forward(self, entries, want) -> Optional[torch.Tensor]:
        table, B = self.table, len(entries)
        if any(len(tok) != 1 for _, tok in entries):
            raise ValueError("the Llama decode step takes one token per sequence")
        if sum(table.blocks_needed(seq, 1) for seq, _ in entries) > table.free_blocks:
            raise OutOfCache("not enough free cache blocks for this step")
        for seq, _ in entries:
            table.extend(seq, 1)
        width = 1
        while width < max(len(seq.blocks) for seq, _ in entries):
            width *= 2
        if (B, width) not in self._buffers:
            self._buffers[B, width] = self.decoder.buffers(B, width)
        buf: DecodeBuffers = self._buffers[B, width]
        i32 = lambda v: torch.tensor(v, dtype=torch.int32)
        buf.ids.copy_(i32([tok[0] for _, tok in entries]))
        buf.positions.copy_(i32([seq.length for seq, _ in entries]))
        buf.seq_used_k.copy_(i32([seq.length + 1 for seq, _ in entries]))
        buf.slot_mapping.copy_(i32([seq.blocks[seq.length // self.BLOCK] * self.BLOCK + seq.length % self.BLOCK for seq, _ in entries]))
        buf.block_table.copy_(i32([seq.blocks + [seq.blocks[-1]] * (width - len(seq.blocks)) for seq, _ in entries]))
        logits = self.decoder.step(buf, self.cache)
        torch.cuda.current_stream(self.device).synchronize()
        for seq, _ in entries:
            table.advance(seq, 1)
        rows = [e for e, places in enumerate(want) if places]
        return logits[rows].float() if rows else None

    def check_health(self) -> None:
        self.decoder.check_health()

    def greedy(self, logits: torch.Tensor) -> List[int]:
        return argmax(logits.to(torch.bfloat16).contiguous()).tolist()     # (the decoder's logits are bf16 to begin with)
