"""Sequence mixers and feed-forwards that hybrid models are put together from.  A mixer reads the normed rows of a step
and writes its f32 output; what it remembers between steps (cache rows, recurrent state) lives in `HybridState`.

Tensor names are relative to the mixer's prefix in the checkpoint."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Tuple

import numpy as np
import torch

from . import _lib
from .dense import Arena, DenseLinear, StepInputs, dtype_code, interleave8
from .layers import GpuWeights, _dev_index, _ptr, _stream

_tables: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}


def rotation_tables(max_pos: int, dims: int, base: float, device) -> Tuple[torch.Tensor, torch.Tensor]:
    """f32 cos / sin [max_pos, dims / 2] of p * base^(-2i/dims), angles formed in f64; one copy per distinct rotation."""
    key = (max_pos, dims, float(base), str(device))
    if key not in _tables:
        freq = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / max(dims, 1))
        ang = np.arange(max_pos, dtype=np.float64)[:, None] * freq[None, :]
        _tables[key] = tuple(torch.from_numpy(f(ang).astype(np.float32)).to(device).contiguous() for f in (np.cos, np.sin))
    return _tables[key]


@dataclass
class StepContext:
    """What every mixer of a step shares."""
    arena: Arena
    inputs: StepInputs
    step: "_lib.Step"
    entries: list                    # (Sequence, number of rows), host side
    block_size: int
    num_blocks: int
    rows: int
    prompt: bool                     # rows of prompts (expanded / chunked kernels) rather than single tokens


class LatentAttention:
    """Multi-head attention whose keys and values come from a low-rank latent; the cache holds the latent and one rotated
    key part per token.  Few rows: attention in the latent space (W_uk folded into the queries, W_uv applied after).
    Prompts in bf16: keys and values are expanded per sequence and a tensor-core prompt kernel runs over them."""

    EXPAND_FROM = 64                 # rows of one sequence from which the expanded form pays

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, eps: float, dtype: torch.dtype, max_pos: int):
        rot = spec["rot"]
        self.heads, self.dim, self.rot_dim = int(spec["heads"]), int(spec["dim"]), int(spec["rot_dim"])
        self.vdim, self.kv_rank, self.q_rank = int(spec["vdim"]), int(spec["kv_rank"]), int(spec["q_rank"])
        self.rot_dims, self.scale, self.eps, self.dtype, self.max_pos = int(rot["dims"]), float(spec["scale"]), float(eps), dtype, max_pos
        take = lambda name: weights.take(f"{prefix}.{name}")
        H, dim, kvr = self.heads, self.dim, self.kv_rank
        self.q_norm, self.kv_norm = take("dq.norm").float(), take("dkv.norm").float()
        self.down = DenseLinear(torch.cat([take("g"), take("dq"), take("dkv")]).to(dtype))
        self.uq = DenseLinear(take("uq").to(dtype))
        uk, uv = take("uk").to(dtype), take("uv").to(dtype)
        self.uk_t = DenseLinear(uk.view(H, dim, kvr).transpose(1, 2).reshape(H * kvr, dim), groups=H)
        self.uv = DenseLinear(uv, groups=H)
        self.uk_rows = DenseLinear(uk)
        self.o = DenseLinear(take("o").to(dtype))
        self.cos, self.sin = rotation_tables(max_pos, self.rot_dims, rot["base"], uk.device)

    @property
    def row_size(self) -> int:
        """Values a token's cache row holds."""
        return self.kv_rank + self.rot_dim

    def shape(self, ctx: StepContext) -> "_lib.LatentShape":
        return _lib.LatentShape(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.q_rank, self.rot_dims, self.max_pos,
                                ctx.block_size, ctx.num_blocks, ctx.inputs.max_blocks, self.eps, self.scale)

    def run(self, ctx: StepContext, h: torch.Tensor, cache: torch.Tensor, y: torch.Tensor) -> None:
        a, T, H, dt = ctx.arena, ctx.rows, self.heads, self.dtype
        lib, c = _lib.models_lib(), _lib.models_context(_dev_index(h.device))
        code, stream, shape, step = dtype_code(dt), _stream(h.device), self.shape(ctx), ctx.step
        ps, pt = ctypes.byref(shape), ctypes.byref(step)
        gate = a.get("la.gate", (T, H * self.vdim), dt)
        low = a.get("la.low", (T, self.q_rank + self.row_size), torch.float32)
        self.down(a, h, gate, y2=low, n_main=H * self.vdim)
        cq = a.get("la.cq", (T, self.q_rank), dt)
        c.check(lib.scr_latent_prepare(c.handle, code, ps, pt, _ptr(low), int(low.stride(0)), _ptr(self.q_norm), _ptr(self.kv_norm),
                                       _ptr(self.cos), _ptr(self.sin), _ptr(cq), _ptr(cache), stream))
        q = a.get("la.q", (T, H * (self.dim + self.rot_dim)), torch.float32)
        self.uq(a, cq, q)
        heads = a.get("la.heads", (T, H * self.vdim), dt)
        if ctx.prompt and dt == torch.bfloat16 and lib.scr_latent_prefill_supported(ps):
            self._expanded(ctx, q, cache, gate, heads)
        else:
            D, kvr = self.row_size, self.kv_rank
            plain = a.get("la.q_plain", (T, H * self.dim), dt)
            ql = a.get("la.q_latent", (T, H * D), dt)
            c.check(lib.scr_latent_queries(c.handle, code, ps, pt, _ptr(q), _ptr(self.cos), _ptr(self.sin), _ptr(plain), H * self.dim,
                                           self.dim, ctypes.c_void_p(ql.data_ptr() + kvr * ql.element_size()), H * D, D, stream))
            self.uk_t(a, plain, ql, x_group=self.dim, y_group=D)
            ol = a.get("la.o_latent", (T, H * kvr), dt)
            need = ctypes.c_size_t(0)
            c.check(lib.scr_latent_attention_workspace(code, ps, pt, ctypes.byref(need)))
            ws = a.get("la.workspace", (need.value,), torch.uint8) if need.value else None
            c.check(lib.scr_latent_attention(c.handle, code, ps, pt, _ptr(ql), _ptr(cache), _ptr(ol), _ptr(ws), need, stream))
            self.uv(a, ol, heads, x_group=kvr, y_group=self.vdim, gate=gate)
        self.o(a, heads, y)

    def _expanded(self, ctx: StepContext, q: torch.Tensor, cache: torch.Tensor, gate: torch.Tensor, heads: torch.Tensor) -> None:
        a, T, H, dt = ctx.arena, ctx.rows, self.heads, self.dtype
        lib, c = _lib.models_lib(), _lib.models_context(_dev_index(q.device))
        stream, shape = _stream(q.device), self.shape(ctx)
        ps, per = ctypes.byref(shape), self.dim + self.rot_dim
        qf = a.get("la.q_full", (T, H * per), dt)
        c.check(lib.scr_latent_queries(c.handle, dtype_code(dt), ps, ctypes.byref(ctx.step), _ptr(q), _ptr(self.cos), _ptr(self.sin), _ptr(qf),
                                       H * per, per, ctypes.c_void_p(qf.data_ptr() + self.dim * qf.element_size()), H * per, per, stream))
        table, row = ctx.inputs.view("table"), 0
        for b, (seq, count) in enumerate(ctx.entries):
            kv = seq.length + count
            ld_v = (kv + 7) // 8 * 8
            lat = a.get("la.latents", (kv, self.kv_rank), dt)
            rot = a.get("la.rotated", (kv, self.rot_dim), dt)
            c.check(lib.scr_latent_gather(c.handle, ps, _ptr(table[b * ctx.inputs.max_blocks:]), kv, _ptr(cache), _ptr(lat), _ptr(rot), stream))
            k = a.get("la.keys", (kv, H * self.dim), dt)
            self.uk_rows(a, lat, k)
            v_t = a.get("la.values_t", (H * self.vdim, ld_v), dt)
            DenseLinear(lat)(a, self.uv.weight, v_t)
            c.check(lib.scr_latent_prefill(c.handle, ps, _ptr(qf[row:]), _ptr(k), _ptr(rot), _ptr(v_t), ld_v, _ptr(gate[row:]),
                                           int(gate.stride(0)), count, seq.length, _ptr(heads[row:]), int(heads.stride(0)), stream))
            row += count


class MatrixMemory:
    """The mLSTM: per head a matrix state, decayed and written with exponential gates; state in f32, one slot per sequence."""

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, eps: float, dtype: torch.dtype):
        self.heads, self.dim, self.vdim = int(spec["heads"]), int(spec["dim"]), int(spec["vdim"])
        self.gate_cap, self.eps, self.dtype = float(spec["gate_cap"]), float(eps), dtype
        take = lambda name: weights.take(f"{prefix}.{name}")
        self.proj = DenseLinear(torch.cat([take(n) for n in ("q", "k", "v", "g", "i", "f")]).to(dtype))
        self.bias_i, self.bias_f, self.norm = take("i.b").float(), take("f.b").float(), take("norm").float()
        self.o = DenseLinear(take("o").to(dtype))

    @property
    def slices(self) -> int:
        return (self.vdim + 31) // 32

    def state(self, slots: int, device) -> Tuple[torch.Tensor, ...]:
        f32, H = torch.float32, self.heads
        return (torch.zeros((slots, H, self.dim, self.vdim), dtype=f32, device=device),
                torch.zeros((slots, H, self.slices, self.dim), dtype=f32, device=device),
                torch.zeros((slots, H, self.slices), dtype=f32, device=device))

    def run(self, ctx: StepContext, h: torch.Tensor, state: Tuple[torch.Tensor, ...], y: torch.Tensor) -> None:
        a, T, H, dt = ctx.arena, ctx.rows, self.heads, self.dtype
        lib, c = _lib.models_lib(), _lib.models_context(_dev_index(h.device))
        code, stream = dtype_code(dt), _stream(h.device)
        shape = _lib.MlstmShape(H, self.dim, self.vdim, self.gate_cap, self.eps)
        qkv = 2 * H * self.dim + H * self.vdim
        n_main = qkv + H * self.vdim
        proj = a.get("mm.proj", (T, n_main), dt)
        gates = a.get("mm.gates", (T, 2 * H), torch.float32)
        self.proj(a, h, proj, y2=gates, n_main=n_main)
        out = a.get("mm.out", (T, H * self.vdim), torch.float32)
        need = ctypes.c_size_t(0)
        c.check(lib.scr_mlstm_workspace(code, ctypes.byref(shape), ctypes.byref(ctx.step), ctypes.byref(need)))
        ws = a.get("mm.workspace", (need.value,), torch.uint8) if need.value else None
        c.check(lib.scr_mlstm_run(c.handle, code, ctypes.byref(shape), ctypes.byref(ctx.step), _ptr(proj), n_main, _ptr(gates), 2 * H,
                                  _ptr(self.bias_i), _ptr(self.bias_f), *(_ptr(t) for t in state), _ptr(out), _ptr(ws), need, stream))
        heads = a.get("mm.heads", (T, H * self.vdim), dt)
        gate = ctypes.c_void_p(proj.data_ptr() + qkv * proj.element_size())
        for r0 in range(0, T, 32768):
            n = min(32768, T - r0)
            c.check(lib.scr_mlstm_finish(c.handle, code, ctypes.byref(shape), _ptr(out[r0:]), _ptr(self.norm),
                                         ctypes.c_void_p(gate.value + r0 * n_main * proj.element_size()), n_main, n, _ptr(heads[r0:]), stream))
        self.o(a, heads, y)


class ClampedGlu:
    """Dense feed-forward with the clamped gated unit a sigmoid(1.702 a) (b + 1)."""

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, dtype: torch.dtype):
        if spec["kind"] != "dense":
            raise ValueError(f"feed-forward kind {spec['kind']!r} is not supported")
        take = lambda name: weights.take(f"{prefix}.{name}")
        gate, up, down = take("gate").to(dtype), take("up").to(dtype), take("down").to(dtype)
        self.gate_up = DenseLinear(interleave8(gate, up), glu_limit=float(spec["limit"]))
        self.ff = self.gate_up.out_features // 2
        if self.ff != down.shape[1]:                       # channels were padded to whole runs of 8
            down = torch.cat([down, torch.zeros((down.shape[0], self.ff - down.shape[1]), dtype=dtype, device=down.device)], 1)
        self.down = DenseLinear(down)

    def run(self, arena: Arena, h: torch.Tensor, y: torch.Tensor) -> None:
        act = arena.get("ff.act", (int(h.shape[0]), self.ff), h.dtype)
        self.gate_up(arena, h, act)
        self.down(arena, act, y)
