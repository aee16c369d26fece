"""Sequence mixers and feed-forwards that hybrid models are put together from.  A mixer reads the normed rows of a step
and writes its f32 output; what it remembers between steps (its `memory`: cache rows, recurrent state) lives in `HybridState`.

`WindowAttention`, `LightningAttention` and `GeluGlu` are for layers that run side by side: they state their input linears as
parts of one matrix (`inputs`), work on its outputs (`run`), and leave their rows for an output linear they share (`o`).

Tensor names are relative to the mixer's prefix in the checkpoint."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, List, Tuple

import numpy as np
import torch

from . import _lib
from .dense import Arena, DenseLinear, JoinedLinear, StepInputs, dtype_code, interleave8
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

    def memory(self, cache_rows: int, slots: int, device) -> torch.Tensor:
        return torch.zeros((cache_rows, self.row_size), dtype=self.dtype, device=device)

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

    def memory(self, cache_rows: int, slots: int, device) -> Tuple[torch.Tensor, ...]:
        return self.state(slots, device)

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


Part = Tuple[str, torch.Tensor, int]                # (name, rows, kind) of a `JoinedLinear`


def distance_buckets(rows: int, far: float) -> List[int]:
    """Row of a `rows`-row bias table for every key distance 0, 1, ... up to the first that takes the last row for good: one
    row per distance in the first half, the others spaced logarithmically up to `far`."""
    half, out = rows // 2, []
    while not out or out[-1] < rows - 1:
        n = len(out)
        if n < half:
            out.append(n)
        elif half == 0 or far <= half:
            out.append(rows - 1)
        else:                                       # (a quotient that is a whole number stays one)
            out.append(min(rows - 1, half + int(np.floor(np.log(n / half) / np.log(far / half) * (rows - half) + 1e-12))))
    return out


def distance_bias(rel: torch.Tensor, far: float) -> Tuple[torch.Tensor, int]:
    """Bias of every head and distance from a table [rows, heads] of buckets, as `scr_window_attention` takes it (in powers of
    two, padded on both sides), and how many distances it has."""
    buckets = distance_buckets(int(rel.shape[0]), far)
    padded = [buckets[0]] * _lib.BIAS_LO + buckets + [buckets[-1]] * _lib.BIAS_HI
    return rel.float()[torch.tensor(padded, device=rel.device)].t().contiguous() * float(np.log2(np.e)), len(buckets)


class WindowAttention:
    """Grouped-head attention over a sliding window and the sequence's first tokens.  Queries and keys pass a short causal
    convolution and an RMS norm over the whole projection, the values are the keys before that norm, a bias per head and
    distance bucket joins the scores, one sigmoid per head gates the output (times `out_scale`).

    The cache holds the values and one f32 per token that turns them into keys (`key_scale`); a slot holds the last projected rows."""

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, eps: float, dtype: torch.dtype, out_scale: float = 1.0):
        self.heads, self.kv_heads, self.dim, self.taps = int(spec["heads"]), int(spec["kv_heads"]), int(spec["dim"]), int(spec["conv"])
        self.window, self.keep_first = int(spec["mask"]["size"]), int(spec["mask"]["keep_first"])
        self.scale, self.out_scale, self.eps, self.dtype, self.prefix = float(spec["scale"]), float(out_scale), float(eps), dtype, prefix
        if self.heads % self.kv_heads:
            raise ValueError(f"{prefix}: {self.heads} heads do not share {self.kv_heads} key/value heads evenly")
        if int(spec["vdim"]) != self.dim:
            raise ValueError(f"{prefix}: values that are keys have their size, not {spec['vdim']}")
        take = lambda name: weights.take(f"{prefix}.{name}")
        self.qk, self.g, self.o = torch.cat([take("q"), take("k")]).to(dtype), take("g").to(dtype), take("o").to(dtype)
        keys = take("k.norm").float().view(self.kv_heads, 1, self.dim).expand(-1, self.heads // self.kv_heads, -1)
        self.norm = (take("q.norm").float() * keys.reshape(-1)).contiguous()       # a query times its head's key weights
        self.conv = torch.cat([take("q.conv"), take("k.conv")]).float().t().contiguous()
        if tuple(self.conv.shape) != (self.taps, self.channels):
            raise ValueError(f"{prefix}: convolution {tuple(self.conv.shape)}, the configuration says {(self.taps, self.channels)}")
        self.bias, self.n_bias = distance_bias(take("rel"), float(spec["bias_max"]))

    @property
    def channels(self) -> int:
        return (self.heads + self.kv_heads) * self.dim

    @property
    def out_features(self) -> int:
        return self.heads * self.dim

    def inputs(self) -> List[Part]:
        return [(f"{self.prefix}.qk", self.qk, _lib.PART_STORE), (f"{self.prefix}.g", self.g, _lib.PART_F32)]

    def buffers(self, ctx: StepContext) -> Dict[str, torch.Tensor]:
        return {f"{self.prefix}.qk": ctx.arena.get("wa.qk", (ctx.rows, self.channels), self.dtype),
                f"{self.prefix}.g": ctx.arena.get("wa.g", (ctx.rows, self.heads), torch.float32)}

    def memory(self, cache_rows: int, slots: int, device) -> Tuple[torch.Tensor, ...]:
        """(values, their scales as keys, projected rows)."""
        return (torch.zeros((cache_rows, self.kv_heads * self.dim), dtype=self.dtype, device=device),
                torch.zeros(cache_rows, dtype=torch.float32, device=device),
                torch.zeros((slots, max(1, self.taps - 1), self.channels), dtype=self.dtype, device=device))

    def shape(self, ctx: StepContext) -> "_lib.WindowShape":
        return _lib.WindowShape(self.heads, self.kv_heads, self.dim, self.taps, self.window, self.keep_first, self.n_bias,
                                ctx.block_size, ctx.num_blocks, ctx.inputs.max_blocks, self.eps, self.scale, self.out_scale)

    def run(self, ctx: StepContext, bufs: Dict[str, torch.Tensor], memory, out: torch.Tensor) -> None:
        """`out`: the gated heads [rows, heads * dim], dense rows of any stride."""
        qk, gate = bufs[f"{self.prefix}.qk"], bufs[f"{self.prefix}.g"]
        cache, inv, rows = memory
        lib, c = _lib.models_lib(), _lib.models_context(_dev_index(qk.device))
        code, stream, ps, pt = dtype_code(self.dtype), _stream(qk.device), ctypes.byref(self.shape(ctx)), ctypes.byref(ctx.step)
        q = ctx.arena.get("wa.q", (ctx.rows, self.heads * self.dim), self.dtype)
        c.check(lib.scr_window_prepare(c.handle, code, ps, pt, _ptr(qk), int(qk.stride(0)), _ptr(self.conv), _ptr(self.norm), _ptr(rows), _ptr(q), _ptr(cache),
                                       _ptr(inv), stream))
        c.check(lib.scr_window_attention(c.handle, code, ps, pt, _ptr(q), _ptr(cache), _ptr(inv), _ptr(self.bias), _ptr(gate), int(gate.stride(0)), _ptr(out),
                                         int(out.stride(0)), stream))


def decay_powers(decay: np.ndarray) -> torch.Tensor:
    """f32 powers 0 .. 64 of every head's decay, and what the decay has beyond its f32 value."""
    powers = decay[:, None] ** np.arange(_lib.DECAY_POWERS - 1)[None, :]
    rest = decay - decay.astype(np.float32).astype(np.float64)
    return torch.from_numpy(np.concatenate([powers, rest[:, None]], 1).astype(np.float32)).contiguous()


class LightningAttention:
    """Linear attention with a constant decay per head: a matrix state in f32, one slot per sequence; the concatenated readouts
    pass one RMS norm and a sigmoid gate (times `out_scale`)."""

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, eps: float, dtype: torch.dtype, out_scale: float = 1.0):
        self.heads, self.dim, self.vdim = int(spec["heads"]), int(spec["dim"]), int(spec["vdim"])
        self.out_scale, self.eps, self.dtype, self.prefix = float(out_scale), float(eps), dtype, prefix
        take = lambda name: weights.take(f"{prefix}.{name}")
        self.qkv = torch.cat([take(n) for n in ("q", "k", "v")]).to(dtype)
        self.g, self.o, self.norm = take("g").to(dtype), take("o").to(dtype), take("norm").float().contiguous()
        decay = np.asarray(spec["decay"], dtype=np.float64)
        if decay.shape != (self.heads,):
            raise ValueError(f"{prefix}: {decay.size} decays for {self.heads} heads")
        self.powers = decay_powers(decay).to(self.norm.device)

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    def inputs(self) -> List[Part]:
        return [(f"{self.prefix}.qkv", self.qkv, _lib.PART_SILU), (f"{self.prefix}.g", self.g, _lib.PART_STORE)]

    def buffers(self, ctx: StepContext) -> Dict[str, torch.Tensor]:
        return {f"{self.prefix}.qkv": ctx.arena.get("li.qkv", (ctx.rows, self.heads * (2 * self.dim + self.vdim)), self.dtype),
                f"{self.prefix}.g": ctx.arena.get("li.g", (ctx.rows, self.out_features), self.dtype)}

    def memory(self, cache_rows: int, slots: int, device) -> torch.Tensor:
        return torch.zeros((slots, self.heads, self.dim, self.vdim), dtype=torch.float32, device=device)

    def run(self, ctx: StepContext, bufs: Dict[str, torch.Tensor], memory: torch.Tensor, out: torch.Tensor) -> None:
        qkv, gate = bufs[f"{self.prefix}.qkv"], bufs[f"{self.prefix}.g"]
        lib, c = _lib.models_lib(), _lib.models_context(_dev_index(qkv.device))
        code, stream = dtype_code(self.dtype), _stream(qkv.device)
        shape = _lib.LightningShape(self.heads, self.dim, self.vdim, self.eps, self.out_scale)
        o = ctx.arena.get("li.out", (ctx.rows, self.out_features), torch.float32)
        need = ctypes.c_size_t(0)
        c.check(lib.scr_lightning_workspace(code, ctypes.byref(shape), ctypes.byref(ctx.step), ctypes.byref(need)))
        ws = ctx.arena.get("li.workspace", (need.value,), torch.uint8) if need.value else None
        c.check(lib.scr_lightning_run(c.handle, code, ctypes.byref(shape), ctypes.byref(ctx.step), _ptr(qkv), int(qkv.stride(0)), _ptr(self.powers), _ptr(memory),
                                      _ptr(o), _ptr(ws), need, stream))
        c.check(lib.scr_lightning_finish(c.handle, code, ctypes.byref(shape), _ptr(o), _ptr(self.norm), _ptr(gate), int(gate.stride(0)), ctx.rows, _ptr(out),
                                         int(out.stride(0)), stream))


class GeluGlu:
    """Dense feed-forward gelu(gate) * up; the activation is an end of its input part."""

    def __init__(self, weights: GpuWeights, prefix: str, spec: dict, dtype: torch.dtype):
        if spec["kind"] != "dense":
            raise ValueError(f"feed-forward kind {spec['kind']!r} is not supported")
        self.prefix = prefix
        take = lambda name: weights.take(f"{prefix}.{name}").to(dtype)
        self.gate_up, self.o = interleave8(take("gate"), take("up")), take("down")
        pad = int(self.gate_up.shape[0]) // 2 - int(self.o.shape[1])
        if pad:                                            # channels were padded to whole runs of 8
            self.o = torch.cat([self.o, torch.zeros((self.o.shape[0], pad), dtype=dtype, device=self.o.device)], 1)

    @property
    def out_features(self) -> int:
        return int(self.o.shape[1])

    def inputs(self) -> List[Part]:
        return [(f"{self.prefix}.act", self.gate_up, _lib.PART_GELU_GLU)]


class SideBySide:
    """Two mixers and, where there is one, a feed-forward over the same input: one matrix before them, one after them, whose sum
    joins the residual.  The mixers' scales are in their `out_scale`."""

    def __init__(self, mixers, mlp=None):
        self.mixers, self.mlp = list(mixers), mlp
        branches = self.mixers + ([mlp] if mlp is not None else [])
        parts = [p for b in reversed(branches) for p in b.inputs()]                  # the feed-forward's pairs first
        self.inp = JoinedLinear(sorted(parts, key=lambda p: p[2] == _lib.PART_F32))  # few, narrow f32 columns last
        self.out = DenseLinear(torch.cat([b.o for b in branches], 1))
        self.columns, at = [], 0
        for b in branches:
            self.columns.append((at, at + b.out_features))
            at += b.out_features
            for name in ("qk", "qkv", "g", "gate_up", "o"):                          # the joined matrices hold them now
                if hasattr(b, name):
                    setattr(b, name, None)

    def memory(self, cache_rows: int, slots: int, device) -> list:
        return [m.memory(cache_rows, slots, device) for m in self.mixers]

    def run(self, ctx: StepContext, h: torch.Tensor, memory: list, residual: torch.Tensor, norm=None) -> None:
        """`residual` += the layer's output; with `norm` (a `TanhNorm`) `h` becomes the norm of the new residual."""
        a = ctx.arena
        rows = a.get("side.rows", (ctx.rows, self.out.in_features), h.dtype)
        bufs = {}
        for m in self.mixers:
            bufs.update(m.buffers(ctx))
        if self.mlp is not None:
            lo, hi = self.columns[-1]
            bufs[f"{self.mlp.prefix}.act"] = rows[:, lo:hi]
        self.inp.run(a, h, bufs)
        for m, mem, (lo, hi) in zip(self.mixers, memory, self.columns):
            m.run(ctx, bufs, mem, rows[:, lo:hi])
        self.out.add_to(a, rows, residual, norm, h)
