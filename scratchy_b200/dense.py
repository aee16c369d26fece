"""Full-precision linears of the sequence models (`scr_dense_linear`), step buffers and the step's device description."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence as Seq, Tuple

import torch

from . import _lib
from .layers import _dev_index, _ptr, _stream

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}
_CODES = {torch.bfloat16: _lib.DTYPE_BF16, torch.float32: _lib.DTYPE_F32}


def dtype_code(dtype: torch.dtype) -> int:
    return _CODES[dtype]


class Arena:
    """Named device buffers of a step.  A buffer grows to the largest size asked for and is then reused, so a step of a
    size that has run before allocates nothing (and can be captured in a CUDA graph)."""

    def __init__(self, device):
        self.device = torch.device(device)
        self._flat: Dict[str, torch.Tensor] = {}

    def get(self, name: str, shape: Seq[int], dtype: torch.dtype) -> torch.Tensor:
        n = 1
        for s in shape:
            n *= int(s)
        nbytes = n * torch.empty((), dtype=dtype).element_size()
        flat = self._flat.get(name)
        if flat is None or flat.numel() < nbytes:
            flat = torch.empty(max(nbytes, 16), dtype=torch.uint8, device=self.device)
            self._flat[name] = flat
        return flat[:nbytes].view(dtype).view(*shape)


class StepInputs:
    """The device description of a step (see include/scratchy_models.h): one int32 buffer holding token ids, positions,
    sequence indices, segments, the rows whose logits are wanted and the block table."""

    def __init__(self, device, rows: int, batch: int, wanted: int, max_blocks: int):
        self.rows, self.batch, self.wanted, self.max_blocks = rows, batch, wanted, max_blocks
        pad = lambda n: (n + 3) // 4 * 4
        sizes = [("ids", rows), ("pos", rows), ("seg", rows), ("segs", 4 * batch), ("want", max(wanted, 1)), ("table", batch * max_blocks)]
        self._at, n = {}, 0
        for name, size in sizes:
            self._at[name] = (n, size)
            n += pad(size)
        self.host = torch.zeros(n, dtype=torch.int32)
        if torch.cuda.is_available():
            self.host = self.host.pin_memory()
        self.buffer = torch.zeros(n, dtype=torch.int32, device=device)

    def view(self, name: str) -> torch.Tensor:
        at, size = self._at[name]
        return self.buffer[at:at + size]

    def fill(self, entries, want: List[int]) -> None:
        """`entries`: (Sequence, token ids) pairs whose blocks are already reserved; `want`: step rows."""
        ids, pos, seg, segs, row = [], [], [], [], 0
        table = torch.zeros((self.batch, self.max_blocks), dtype=torch.int32)
        self.max_count = self.max_kv = 0
        for b, (seq, tokens) in enumerate(entries):
            n = len(tokens)
            ids += tokens
            pos += range(seq.length, seq.length + n)
            seg += [b] * n
            segs += [row, n, seq.length, seq.slot]
            table[b, :len(seq.blocks)] = torch.tensor(seq.blocks, dtype=torch.int32)
            row += n
            self.max_count, self.max_kv = max(self.max_count, n), max(self.max_kv, seq.length + n)
        for name, values in (("ids", ids), ("pos", pos), ("seg", seg), ("segs", segs), ("want", want or [0])):
            at, size = self._at[name]
            if len(values) != size:
                raise ValueError(f"step description: {len(values)} values for `{name}`, expected {size}")
            self.host[at:at + size] = torch.tensor(values, dtype=torch.int32)
        at, size = self._at["table"]
        self.host[at:at + size] = table.reshape(-1)
        self.buffer.copy_(self.host, non_blocking=True)

    def struct(self, num_slots: int, max_kv: Optional[int] = None) -> _lib.Step:
        return _lib.Step(self.view("seg").data_ptr(), self.view("pos").data_ptr(), self.view("segs").data_ptr(),
                         self.view("table").data_ptr(), self.rows, self.batch, self.max_count, max_kv or self.max_kv, num_slots)


def interleave8(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Rows of a fused gate/up matrix: per 16, 8 gate rows then the 8 up rows of the same channels; the channel count is
    padded to a multiple of 8 with zero rows (whose activation is zero)."""
    n = gate.shape[0]
    pad = (-n) % 8
    if pad:
        zeros = torch.zeros((pad, gate.shape[1]), dtype=gate.dtype, device=gate.device)
        gate, up = torch.cat([gate, zeros]), torch.cat([up, zeros])
    n += pad
    return torch.stack([gate.reshape(n // 8, 8, -1), up.reshape(n // 8, 8, -1)], dim=1).reshape(2 * n, -1).contiguous()


@dataclass
class DenseLinear:
    """y = x W^T with W [groups * N, K] in the activation dtype."""
    weight: torch.Tensor
    groups: int = 1
    glu_limit: Optional[float] = None        # set: a fused gate/up matrix (`interleave8`) with the clamped activation
    glu_alpha: float = 1.702

    def __post_init__(self):
        self.weight = self.weight.contiguous()
        if self.weight.shape[0] % self.groups:
            raise ValueError("rows are not a multiple of the groups")

    @property
    def out_features(self) -> int:
        return int(self.weight.shape[0]) // self.groups

    @property
    def in_features(self) -> int:
        return int(self.weight.shape[1])

    def __call__(self, arena: Arena, x: torch.Tensor, y: torch.Tensor, *, y2: Optional[torch.Tensor] = None, n_main: Optional[int] = None,
                 gate: Optional[torch.Tensor] = None, rows: Optional[int] = None, ldx: Optional[int] = None, x_group: int = 0,
                 ldy: Optional[int] = None, y_group: int = 0) -> torch.Tensor:
        """x, y, y2, gate: 2-D with dense rows unless strides are given (`ldx`, `x_group`, ... in elements)."""
        w = self.weight
        code, M = dtype_code(w.dtype), int(x.shape[0]) if rows is None else rows
        d = _lib.Dense(w.data_ptr(), x.data_ptr(), y.data_ptr(), 0 if y2 is None else y2.data_ptr(), 0 if gate is None else gate.data_ptr(),
                       int(x.stride(0)) if ldx is None else ldx, x_group, int(y.stride(0)) if ldy is None else ldy, y_group,
                       0 if y2 is None else int(y2.stride(0)), 0 if gate is None else int(gate.stride(0)), M, self.out_features,
                       self.in_features, self.groups, self.out_features if n_main is None else n_main,
                       int(y.dtype == torch.float32 and w.dtype != torch.float32), int(self.glu_limit is not None),
                       self.glu_limit if self.glu_limit is not None else 0.0, self.glu_alpha)
        self._launch(arena, code, d)
        return y

    def _launch(self, arena: Arena, code: int, d: "_lib.Dense") -> None:
        w = self.weight
        lib, ctx = _lib.models_lib(), _lib.models_context(_dev_index(w.device))
        need = ctypes.c_size_t(0)
        ctx.check(lib.scr_dense_workspace_size(code, d.M, d.N, d.K, self.groups, ctypes.byref(need)))
        ws = arena.get("dense.workspace", (need.value,), torch.uint8) if need.value else None
        ctx.check(lib.scr_dense_linear(ctx.handle, code, ctypes.byref(d), _ptr(ws), need, _stream(w.device)))

    def add_to(self, arena: Arena, x: torch.Tensor, residual: torch.Tensor, norm: Optional["TanhNorm"] = None,
               out: Optional[torch.Tensor] = None) -> None:
        """residual (f32) += x W^T, and with `norm` the norm of the new residual into `out`."""
        d = _lib.Dense(self.weight.data_ptr(), x.data_ptr(), 0 if norm is None else out.data_ptr(), 0, 0, int(x.stride(0)), 0,
                       0 if norm is None else int(out.stride(0)), 0, 0, 0, int(x.shape[0]), self.out_features, self.in_features, 1, self.out_features)
        d.residual, d.ld_residual = residual.data_ptr(), int(residual.stride(0))
        if norm is not None:
            d.tanh_w, d.tanh_b, d.tanh_alpha = norm.w.data_ptr(), norm.b.data_ptr(), norm.alpha
        self._launch(arena, dtype_code(self.weight.dtype), d)


class JoinedLinear(DenseLinear):
    """Several linears of one input as one matrix.  `parts`: (name, rows, kind) in order of their columns; a gate/up pair
    (`interleave8`) comes first or after a multiple of 16 columns."""

    def __init__(self, parts: Seq[Tuple[str, torch.Tensor, int]]):
        super().__init__(torch.cat([w for _, w, _ in parts]))
        self.parts, n = {}, 0
        for name, w, kind in parts:
            n += int(w.shape[0])
            self.parts[name] = (n, kind)

    def run(self, arena: Arena, x: torch.Tensor, outs: Dict[str, torch.Tensor]) -> None:
        """`outs`: a 2-D tensor with dense rows for every part."""
        d = _lib.Dense(self.weight.data_ptr(), x.data_ptr())
        d.ldx, d.M, d.N, d.K, d.groups, d.n_main = int(x.stride(0)), int(x.shape[0]), self.out_features, self.in_features, 1, self.out_features
        d.n_parts = len(self.parts)
        for p, (name, (n_end, kind)) in enumerate(self.parts.items()):
            d.parts[p] = _lib.DensePart(outs[name].data_ptr(), int(outs[name].stride(0)), n_end, kind)
        self._launch(arena, dtype_code(self.weight.dtype), d)


@dataclass
class TanhNorm:
    """Dynamic tanh in place of a norm: tanh(alpha x) * w + b."""
    alpha: float
    w: torch.Tensor
    b: torch.Tensor

    @classmethod
    def take(cls, weights, name: str) -> "TanhNorm":
        return cls(float(weights.take(f"{name}.alpha").float().reshape(())), weights.take(name).float().contiguous(),
                   weights.take(f"{name}.b").float().contiguous())


def seq_embed(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, raw: Optional[torch.Tensor] = None) -> None:
    """x (f32 residual) = table[ids]; `raw`: the rows as stored (dense rows, any stride)."""
    ctx = _lib.models_context(_dev_index(table.device))
    ctx.check(_lib.models_lib().scr_seq_embed(ctx.handle, dtype_code(table.dtype), _ptr(ids), int(x.shape[0]), _ptr(table),
                                              int(table.shape[0]), int(table.shape[1]), _ptr(x), _ptr(raw),
                                              0 if raw is None else int(raw.stride(0)), _stream(table.device)))


def seq_norm(x: torch.Tensor, eps: float, *, delta: Optional[torch.Tensor] = None, w_delta: Optional[torch.Tensor] = None,
             bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None, w_out: Optional[torch.Tensor] = None,
             row_index: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None, tanh: Optional[TanhNorm] = None) -> None:
    """The step between two sublayers on the f32 residual (`scr_seq_norm`); `tanh` in place of `w_out`."""
    if tanh is not None:
        w_out = tanh.w
    rows = int(x.shape[0]) if row_index is None else int(row_index.shape[0])
    a = _lib.SeqNorm(x.data_ptr(), *(0 if t is None else t.data_ptr() for t in (delta, w_delta, bias, w_out, out, row_index)),
                     0 if out is None else int(out.stride(0)), rows, int(x.shape[0]), int(x.shape[1]), eps, 0 if tanh is None else tanh.b.data_ptr(), 0.0 if tanh is None else tanh.alpha)
    ctx = _lib.models_context(_dev_index(x.device))
    ctx.check(_lib.models_lib().scr_seq_norm(ctx.handle, dtype_code(out_dtype or (torch.float32 if out is None else out.dtype)),
                                             ctypes.byref(a), _stream(x.device)))


def greedy(logits: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Greedy token per row of f32 logits: largest value, smallest id among equals."""
    if out is None:
        out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    ctx = _lib.models_context(_dev_index(logits.device))
    ctx.check(_lib.models_lib().scr_seq_argmax(ctx.handle, _ptr(logits), int(logits.stride(0)), int(logits.shape[0]), int(logits.shape[1]),
                                               _ptr(out), _stream(logits.device)))
    return out
