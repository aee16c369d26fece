"""Every mechanism of the sequence models on its own, against the plain statement: linears with their ends, embedding,
norms, rotation, latent attention in each of its forms, the recurrence token by token and in chunks, greedy sampling."""
import ctypes

import numpy as np
import pytest

from oracle import sequence_plain as plain
from tests import seq_util as su

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TOL = {"float32": 2e-6, "bfloat16": 4e-3}


def torch_():
    import torch
    return torch


def dev(x, dtype="float32"):
    torch = torch_()
    return torch.from_numpy(np.ascontiguousarray(x, np.float32)).cuda().to(getattr(torch, dtype))


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def draw(rng, shape, dtype, gain=1.0):
    x = (gain * rng.standard_normal(shape)).astype(np.float32)
    return su.round_bf16(x) if dtype == "bfloat16" else x


def arena():
    from scratchy_b200.dense import Arena
    return Arena("cuda")


def lib():
    from scratchy_b200 import _lib
    return _lib.models_lib(), _lib.models_context(0)


def ptr(t, offset=0):
    return ctypes.c_void_p(t.data_ptr() + offset * t.element_size())


def stream():
    return ctypes.c_void_p(torch_().cuda.current_stream().cuda_stream)


def healthy():
    lib()[1].device_status(None)


# ------------------------------------------------------------------------------------------------ linears
SHAPES = [(1, 48, 40), (1, 4096, 1536), (2, 17, 200), (8, 130, 72), (9, 96, 64), (16, 640, 1032), (17, 100, 88), (40, 256, 3072), (130, 300, 96),
          (300, 520, 136), (1, 5, 9), (20, 33, 13), (600, 1000, 520)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear(M, N, K, dtype):
    from scratchy_b200.dense import DenseLinear
    torch = torch_()
    rng = np.random.default_rng(M * N + K)
    x, w = draw(rng, (M, K), dtype), draw(rng, (N, K), dtype)
    want = x.astype(np.float64) @ w.astype(np.float64).T
    a, lin, xd = arena(), DenseLinear(dev(w, dtype)), dev(x, dtype)
    y = torch.full((M, N), float("nan"), dtype=torch.float32, device="cuda")
    lin(a, xd, y)
    assert su.rel(host(y), want) < (3e-6 if dtype == "float32" else 1e-5)      # f32 sums under both
    y = torch.full((M, N), float("nan"), dtype=getattr(torch, dtype), device="cuda")
    lin(a, xd, y)
    assert su.rel(host(y), want) < TOL[dtype]
    n_main = N // 3
    y, y2 = torch.full((M, n_main + 3), 7.0, dtype=getattr(torch, dtype), device="cuda"), torch.full((M, N - n_main), 7.0, device="cuda")
    lin(a, xd, y, y2=y2, n_main=n_main)
    if n_main:
        assert su.rel(host(y)[:, :n_main], want[:, :n_main]) < TOL[dtype] and (host(y)[:, n_main:] == 7.0).all()
    assert su.rel(host(y2), want[:, n_main:]) < 1e-5
    healthy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 48, 24), (5, 2, 16, 128), (16, 4, 40, 64), (33, 3, 24, 48), (200, 5, 136, 72), (3, 2, 7, 10)])
def test_linear_in_groups_with_an_output_gate(M, H, N, K, dtype):
    """One weight block per head; outputs interleaved into rows that hold more than the sums, and the sigmoid gate."""
    from scratchy_b200.dense import DenseLinear
    torch = torch_()
    rng = np.random.default_rng(M + H + N + K)
    x, w, g = draw(rng, (M, H, K), dtype), draw(rng, (H, N, K), dtype, K ** -0.5), draw(rng, (M, H * N), dtype)
    want = np.einsum("mhk,hnk->mhn", x.astype(np.float64), w.astype(np.float64))
    lin, a = DenseLinear(dev(w.reshape(H * N, K), dtype), groups=H), arena()
    pad = N + 8
    y = torch.full((M, H * pad), 7.0, dtype=getattr(torch, dtype), device="cuda")
    lin(a, dev(x.reshape(M, H * K), dtype), y, x_group=K, y_group=pad)
    got = host(y).reshape(M, H, pad)
    assert su.rel(got[:, :, :N], want) < TOL[dtype] and (got[:, :, N:] == 7.0).all()
    y = torch.empty((M, H * N), dtype=getattr(torch, dtype), device="cuda")
    lin(a, dev(x.reshape(M, H * K), dtype), y, x_group=K, y_group=N, gate=dev(g, dtype))
    assert su.rel(host(y), want.reshape(M, H * N) * plain.sigmoid(g.astype(np.float64))) < TOL[dtype]
    healthy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 7, 16, 50, 200])
@pytest.mark.parametrize("ff,K,limit", [(72, 88, 0.8), (10, 40, 2.5), (520, 256, 1.0)])
def test_gate_and_up_with_the_clamped_unit(M, ff, K, limit, dtype):
    from scratchy_b200.dense import DenseLinear, interleave8
    torch = torch_()
    rng = np.random.default_rng(M + ff)
    x, g, u = draw(rng, (M, K), dtype), draw(rng, (ff, K), dtype, 2 * K ** -0.5), draw(rng, (ff, K), dtype, 2 * K ** -0.5)
    x64 = x.astype(np.float64)
    want = plain.clamped_glu(x64 @ g.astype(np.float64).T, x64 @ u.astype(np.float64).T, limit)
    assert (np.abs(x64 @ u.astype(np.float64).T) > limit).any()                  # the clamp is at work
    lin = DenseLinear(interleave8(dev(g, dtype), dev(u, dtype)), glu_limit=limit)
    y = torch.full((M, (ff + 7) // 8 * 8), float("nan"), dtype=getattr(torch, dtype), device="cuda")
    lin(arena(), dev(x, dtype), y)
    assert su.rel(host(y)[:, :ff], want) < TOL[dtype] and not host(y)[:, ff:].any()
    healthy()


# ------------------------------------------------------------------------------------------------ rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [88, 90, 256, 3072, 3])
def test_norms_between_sublayers(W, dtype):
    from scratchy_b200.dense import seq_norm
    torch = torch_()
    rng = np.random.default_rng(W)
    T, eps = 5, 0.01
    x, d = rng.standard_normal((T, W)).astype(np.float32), 3 * rng.standard_normal((T, W)).astype(np.float32)
    wd, wo, bias = (0.5 * rng.standard_normal(W).astype(np.float32) for _ in range(3))
    for delta, w_delta, b in ((None, None, None), (d, wd, None), (d, None, bias), (d, None, None)):
        xd = dev(x)
        out = torch.full((T, W + 4), 7.0, dtype=getattr(torch, dtype), device="cuda")
        seq_norm(xd, eps, delta=None if delta is None else dev(delta), w_delta=None if w_delta is None else dev(w_delta),
                 bias=None if b is None else dev(b), out=out, w_out=dev(wo))
        want_x = x.astype(np.float64)
        if w_delta is not None:
            want_x = want_x + plain.norm_around_zero(d.astype(np.float64), wd, eps)
        elif delta is not None:
            want_x = d.astype(np.float64) + (0 if b is None else b)
        assert su.rel(host(xd), want_x) < 1e-6
        assert su.rel(host(out)[:, :W], plain.norm_around_zero(want_x, wo, eps)) < TOL[dtype] and (host(out)[:, W:] == 7.0).all()
    out = torch.empty((T, W), dtype=getattr(torch, dtype), device="cuda")
    seq_norm(dev(x), eps, out=out)                                               # the row itself
    assert su.rel(host(out), x) < TOL[dtype]
    rows = torch.tensor([4, 0, 0, 2], dtype=torch.int32, device="cuda")
    out = torch.empty((4, W), dtype=getattr(torch, dtype), device="cuda")
    seq_norm(dev(x), eps, out=out, w_out=dev(wo), row_index=rows)
    assert su.rel(host(out), plain.norm_around_zero(x.astype(np.float64), wo, eps)[[4, 0, 0, 2]]) < TOL[dtype]
    healthy()


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_and_greedy_sampling(dtype):
    from scratchy_b200 import _lib
    from scratchy_b200.dense import greedy, seq_embed
    torch = torch_()
    rng = np.random.default_rng(3)
    table = draw(rng, (40, 54), dtype)
    ids = torch.tensor([0, 39, 7, 7], dtype=torch.int32, device="cuda")
    x, cat = torch.empty((4, 54), device="cuda"), torch.full((4, 108), 7.0, dtype=getattr(torch, dtype), device="cuda")
    seq_embed(ids, dev(table, dtype), x, cat[:, 54:])
    assert np.array_equal(host(x), table[[0, 39, 7, 7]]) and np.array_equal(host(cat)[:, 54:], table[[0, 39, 7, 7]]) and (host(cat)[:, :54] == 7.0).all()
    logits = torch.zeros((4, 1234), device="cuda")
    logits[0, 17] = logits[0, 900] = 2.0
    logits[1, 1233] = 1e-3
    logits[2, :] = float("nan")
    logits[2, 5] = -3.0
    assert greedy(logits).tolist() == [17, 1233, 5, 0]
    seq_embed(torch.tensor([40], dtype=torch.int32, device="cuda"), dev(table, dtype), x[:1])
    with pytest.raises(_lib.ScratchyCudaError):
        healthy()
    assert not host(x[:1]).any()


# ------------------------------------------------------------------------------------------------ latent attention
class Latents:
    """A paged latent cache on the device with scattered blocks, its rows in host memory, and the step structures."""

    def __init__(self, m, lengths, counts, dtype, seed, block_size=16, max_pos=4096):
        from scratchy_b200 import _lib
        from scratchy_b200.mixers import rotation_tables
        torch = torch_()
        self.m, self.dtype, rng = m, dtype, np.random.default_rng(seed)
        self.rng, self.counts, self.D = rng, counts, m["kv_rank"] + m["rot_dim"]
        totals = [a + n for a, n in zip(lengths, counts)]
        self.max_blocks = max(-(-t // block_size) for t in totals)
        need = sum(-(-t // block_size) for t in totals)
        self.num_blocks = need + 3
        perm = rng.permutation(self.num_blocks)
        table, at, self.rows = np.full((len(counts), self.max_blocks), -1, np.int32), 0, []
        cache = np.full((self.num_blocks * block_size, self.D), np.nan, np.float32)       # unowned rows must not be read
        self.slots = []
        for b, t in enumerate(totals):
            n = -(-t // block_size)
            table[b, :n] = perm[at:at + n]
            at += n
            slot = (table[b, np.arange(t) // block_size].astype(np.int64) * block_size + np.arange(t) % block_size)
            rows = draw(rng, (t, self.D), dtype)
            cache[slot] = rows
            self.rows.append(rows)
            self.slots.append(slot)
        self.cache = dev(cache, dtype)
        self.positions = np.concatenate([np.arange(a, a + n) for a, n in zip(lengths, counts)])
        self.T = int(sum(counts))
        seg = np.concatenate([[b] * n for b, n in enumerate(counts)])
        first = np.cumsum([0] + list(counts[:-1]))
        segs = np.stack([first, counts, lengths, np.arange(len(counts))], 1)
        i32 = lambda x: torch.from_numpy(np.ascontiguousarray(x, np.int32)).cuda()
        self.dev_arrays = [i32(seg), i32(self.positions), i32(segs), i32(table)]
        self.first = first
        self.shape = _lib.LatentShape(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["rot"]["dims"], max_pos,
                                      block_size, self.num_blocks, self.max_blocks, 1e-5, m["scale"])
        self.step = _lib.Step(*[a.data_ptr() for a in self.dev_arrays], self.T, len(counts), max(counts), max(totals), len(counts))
        self.cos, self.sin = rotation_tables(max_pos, m["rot"]["dims"], m["rot"]["base"], "cuda")
        self.lengths = lengths

    def code(self):
        from scratchy_b200.dense import dtype_code
        return dtype_code(getattr(torch_(), self.dtype))


def run_latent(lt, q):
    """q [T, heads, D] host -> [T, heads, kv_rank] from scr_latent_attention."""
    torch = torch_()
    L, c = lib()
    qd = dev(q, lt.dtype)
    out = torch.full((lt.T, lt.m["heads"], lt.m["kv_rank"]), float("nan"), dtype=getattr(torch, lt.dtype), device="cuda")
    need = ctypes.c_size_t(0)
    c.check(L.scr_latent_attention_workspace(lt.code(), ctypes.byref(lt.shape), ctypes.byref(lt.step), ctypes.byref(need)))
    ws = torch.empty(max(16, need.value), dtype=torch.uint8, device="cuda")
    c.check(L.scr_latent_attention(c.handle, lt.code(), ctypes.byref(lt.shape), ctypes.byref(lt.step), ptr(qd), ptr(lt.cache), ptr(out), ptr(ws),
                                   need, stream()))
    healthy()
    return host(out)


def plain_latent(lt, q):
    kvr, out, row = lt.m["kv_rank"], np.zeros((lt.T, lt.m["heads"], lt.m["kv_rank"])), 0
    for b, n in enumerate(lt.counts):
        rows = lt.rows[b].astype(np.float64)
        for i in range(n):
            seen = rows[:lt.lengths[b] + i + 1]
            s = q[row].astype(np.float64) @ seen.T * lt.m["scale"]
            p = np.exp(s - s.max(1, keepdims=True))
            out[row] = (p / p.sum(1, keepdims=True)) @ seen[:, :kvr]
            row += 1
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_rank,rot_dim", [(3, 48, 8), (1, 64, 16), (24, 512, 64), (16, 104, 24), (5, 256, 32), (40, 136, 8), (2, 12, 6)])
@pytest.mark.parametrize("lengths,counts", [([0], [1]), ([63], [1]), ([300], [1]), ([0, 130, 64, 700], [1, 1, 1, 1]), ([5, 0, 90], [9, 3, 20])])
def test_latent_attention_over_the_paged_cache(heads, kv_rank, rot_dim, lengths, counts, dtype):
    m = su.attention_spec(heads=heads, kv_rank=kv_rank, rot_dim=rot_dim, scale=(kv_rank + rot_dim) ** -0.5)["mixer"]
    lt = Latents(m, lengths, counts, dtype, seed=heads + kv_rank)
    q = draw(lt.rng, (lt.T, heads, lt.D), dtype)
    assert su.rel(run_latent(lt, q), plain_latent(lt, q)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_key_among_hundreds_is_found_wherever_it_sits(dtype):
    """A key that outweighs all others, at the ends of pages and tiles and at either end of the sequence; a key of the future
    that would outweigh everything stays unseen."""
    kvr, H = 64, 4
    m = su.attention_spec(heads=H, kv_rank=kvr, rot_dim=16, scale=0.125)["mixer"]
    for at in (0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 500, 511):
        lt = Latents(m, [510], [3], dtype, seed=at)
        rows, q = lt.rows[0], draw(lt.rng, (3, H, lt.D), dtype)
        rows[at] = su.round_bf16(4.0 * q[:, 1].sum(0))                               # a score around 4 * 80 / 8
        rows[512] = su.round_bf16(9.0 * q[:, 1].sum(0))                              # position 512: the last row's own
        lt.cache[torch_().from_numpy(lt.slots[0]).cuda()] = dev(rows, dtype)
        got, want = run_latent(lt, q), plain_latent(lt, q)
        assert su.rel(got, want) < TOL[dtype]
        visible = [i for i in range(3) if at <= 510 + i]
        for i in visible:
            mine = rows[512] if i == 2 else rows[at]
            assert su.rel(want[i, 1], mine[:kvr]) < 0.05                             # the far key is what comes out
            assert su.rel(got[i, 1], mine[:kvr]) < 0.05


@pytest.mark.parametrize("dim,rot_dim,vdim,heads,kv_rank", [(64, 16, 64, 2, 64), (24, 8, 40, 3, 48), (128, 64, 128, 2, 512), (128, 32, 104, 1, 128),
                                                            (192, 64, 16, 2, 64), (8, 8, 8, 3, 16)])
@pytest.mark.parametrize("pos0,rows", [(0, 1), (0, 64), (0, 129), (0, 300), (37, 100), (500, 257), (127, 2)])
def test_expanded_prompt_attention(dim, rot_dim, vdim, heads, kv_rank, pos0, rows):
    torch = torch_()
    L, c = lib()
    m = su.attention_spec(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank)["mixer"]
    lt = Latents(m, [pos0], [rows], "bfloat16", seed=pos0 + rows + dim)
    assert L.scr_latent_prefill_supported(ctypes.byref(lt.shape)) == 1
    kv, rng, dt = pos0 + rows, lt.rng, "bfloat16"
    q, k, r, v = draw(rng, (rows, heads, dim + rot_dim), dt, 2.0), draw(rng, (kv, heads, dim), dt), draw(rng, (kv, rot_dim), dt), draw(rng, (kv, heads, vdim), dt)
    far = (kv // 2) // 64 * 64                                                         # a key at a tile's start that outweighs the others for head 0
    k[far, 0] = su.round_bf16(3.0 * q[-1, 0, :dim])
    g = draw(rng, (rows, heads * vdim), dt)
    ld_v = (kv + 7) // 8 * 8
    vt = np.full((heads * vdim, ld_v), np.nan, np.float32)                             # columns past the keys are never read
    vt[:, :kv] = v.reshape(kv, heads * vdim).T
    out = torch.full((rows, heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
    args = [dev(t, dt) for t in (q, k, r, vt, g)]
    c.check(L.scr_latent_prefill(c.handle, ctypes.byref(lt.shape), *[ptr(t) for t in args[:4]], ld_v, ptr(args[4]), heads * vdim, rows, pos0, ptr(out),
                                 heads * vdim, stream()))
    healthy()
    want = np.zeros((rows, heads, vdim))
    for h in range(heads):
        s = (q[:, h, :dim].astype(np.float64) @ k[:, h].astype(np.float64).T + q[:, h, dim:].astype(np.float64) @ r.astype(np.float64).T) * m["scale"]
        s = np.where(np.arange(kv)[None, :] <= pos0 + np.arange(rows)[:, None], s, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        want[:, h] = (p / p.sum(1, keepdims=True)) @ v[:, h].astype(np.float64)
    want = want.reshape(rows, -1) * plain.sigmoid(g.astype(np.float64))
    assert su.rel(host(out), want) < TOL[dt]
    assert np.abs(host(out) - want).max() < 0.03 * np.abs(want).max()


def test_scores_that_climb_along_the_sequence_rescale_the_sums():
    """Keys ordered so that the running maximum grows at every tile by more than the kernels let it grow unscaled."""
    torch = torch_()
    L, c = lib()
    dim, rot, vdim, rows = 64, 8, 64, 256
    m = su.attention_spec(heads=1, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=64, scale=1.0)["mixer"]
    lt = Latents(m, [0], [rows], "bfloat16", seed=1)
    rng = lt.rng
    q, k = np.zeros((rows, 1, dim + rot), np.float32), np.zeros((rows, 1, dim), np.float32)
    q[:, 0, 0] = 1.0
    k[:, 0, 0] = su.round_bf16(np.arange(rows) / 4.0)                                  # 16 per tile of 64: e^16 between tiles
    r, v, g = np.zeros((rows, rot), np.float32), draw(rng, (rows, vdim), "bfloat16"), np.full((rows, vdim), 30.0, np.float32)
    out = torch.empty((rows, vdim), dtype=torch.bfloat16, device="cuda")
    args = [dev(t, "bfloat16") for t in (q, k, r, v.T.copy(), g)]
    c.check(L.scr_latent_prefill(c.handle, ctypes.byref(lt.shape), *[ptr(t) for t in args[:4]], rows, ptr(args[4]), vdim, rows, 0, ptr(out), vdim, stream()))
    healthy()
    s = np.where(np.tril(np.ones((rows, rows), bool)), k[:, 0, 0].astype(np.float64)[None, :], -np.inf)
    p = np.exp(s - s.max(1, keepdims=True))
    assert su.rel(host(out), (p / p.sum(1, keepdims=True)) @ v.astype(np.float64)) < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot_dim,rot_dims,base", [(8, 8, 700.0), (16, 12, 1e6), (2, 2, 10.0), (6, 4, 1.0)])
def test_latent_rows_and_rotated_queries(rot_dim, rot_dims, base, dtype):
    torch = torch_()
    L, c = lib()
    m = su.attention_spec(heads=3, rot_dim=rot_dim, rot_dims=rot_dims, base=base)["mixer"]
    lt = Latents(m, [0, 15, 2000], [3, 2, 1], dtype, seed=5)
    rng, H, dim, kvr, qr = lt.rng, 3, m["dim"], m["kv_rank"], m["q_rank"]
    d = rng.standard_normal((lt.T, qr + kvr + rot_dim + 1)).astype(np.float32)         # a row stride of its own
    wq, wkv = rng.standard_normal(qr).astype(np.float32), rng.standard_normal(kvr).astype(np.float32)
    cq = torch.empty((lt.T, qr), dtype=getattr(torch, dtype), device="cuda")
    dd, args = dev(d), [dev(wq), dev(wkv)]
    c.check(L.scr_latent_prepare(c.handle, lt.code(), ctypes.byref(lt.shape), ctypes.byref(lt.step), ptr(dd), d.shape[1], ptr(args[0]), ptr(args[1]),
                                 ptr(lt.cos), ptr(lt.sin), ptr(cq), ptr(lt.cache), stream()))
    d64 = d.astype(np.float64)
    assert su.rel(host(cq), plain.unit_rms(d64[:, :qr], 1e-5) * wq) < TOL[dtype]
    want = np.concatenate([plain.unit_rms(d64[:, qr:qr + kvr], 1e-5) * wkv,
                           plain.rotate_interleaved(d64[:, qr + kvr:-1], lt.positions, rot_dims, base)], 1)
    slots = np.concatenate([lt.slots[b][lt.lengths[b]:] for b in range(3)])
    cache = host(lt.cache)
    assert su.rel(cache[slots], want) < max(TOL[dtype], 2e-5)
    for b in range(3):                                                                 # what was there before is untouched
        assert np.array_equal(cache[lt.slots[b][:lt.lengths[b]]], lt.rows[b][:lt.lengths[b]].astype(np.float64))
    q = rng.standard_normal((lt.T, H, dim + rot_dim)).astype(np.float32)
    qp, qt = (torch.full((lt.T, H, dim + rot_dim), 7.0, dtype=getattr(torch, dtype), device="cuda") for _ in range(2))
    qd, per = dev(q), dim + rot_dim
    c.check(L.scr_latent_queries(c.handle, lt.code(), ctypes.byref(lt.shape), ctypes.byref(lt.step), ptr(qd), ptr(lt.cos), ptr(lt.sin), ptr(qp), H * per, per,
                                 ptr(qt, dim), H * per, per, stream()))
    healthy()
    assert su.rel(host(qp)[:, :, :dim], q[:, :, :dim]) < TOL[dtype] and (host(qp)[:, :, dim:] == 7.0).all()
    assert su.rel(host(qt)[:, :, dim:], plain.rotate_interleaved(q[:, :, dim:].astype(np.float64), lt.positions, rot_dims, base)) < max(TOL[dtype], 2e-5)


# ------------------------------------------------------------------------------------------------ the recurrence
def draw_memory(rng, T, m, dtype):
    """Projections whose keys lean towards the queries (n.q is not all noise)."""
    p, qk = rng.standard_normal((T, 2 * m["heads"] * m["dim"] + m["heads"] * m["vdim"])).astype(np.float32), m["heads"] * m["dim"]
    p[:, qk:2 * qk] = 0.8 * p[:, :qk] + 0.6 * p[:, qk:2 * qk]
    return su.round_bf16(p) if dtype == "bfloat16" else p


def run_memory(m, dtype, proj, gates, bi, bf, portions, slots, state=None):
    """Runs the rows of each sequence in the given portions; returns readouts per sequence and the state."""
    from scratchy_b200 import _lib
    from scratchy_b200.dense import dtype_code
    torch = torch_()
    L, c = lib()
    H, dim, vdim, B = m["heads"], m["dim"], m["vdim"], len(proj)
    shape, sl, total = _lib.MlstmShape(H, dim, vdim, m["gate_cap"], 1e-5), (vdim + 31) // 32, max(slots) + 1
    if state is None:
        state = (torch.full((total, H, dim, vdim), float("nan"), device="cuda"), torch.full((total, H, sl, dim), float("nan"), device="cuda"),
                 torch.full((total, H, sl), float("nan"), device="cuda"))             # a fresh sequence ignores what the slot holds
    outs, at = [[] for _ in range(B)], [0] * B
    bid, bfd = dev(bi), dev(bf)
    for step in portions:
        counts = [min(n, len(proj[b]) - at[b]) for b, n in enumerate(step)]
        who = [b for b in range(B) if counts[b] > 0]
        if not who:
            break
        p = np.concatenate([proj[b][at[b]:at[b] + counts[b]] for b in who])
        g = np.concatenate([gates[b][at[b]:at[b] + counts[b]] for b in who])
        first = np.cumsum([0] + [counts[b] for b in who])[:-1]
        segs = torch.from_numpy(np.array([[f, counts[b], at[b], slots[b]] for f, b in zip(first, who)], np.int32)).cuda()
        st = _lib.Step(0, 0, segs.data_ptr(), 0, len(p), len(who), max(counts), 0, total)
        pd, gd, out = dev(p, dtype), dev(g), torch.full((len(p), H * vdim), float("nan"), device="cuda")
        need = ctypes.c_size_t(0)
        c.check(L.scr_mlstm_workspace(dtype_code(getattr(torch, dtype)), ctypes.byref(shape), ctypes.byref(st), ctypes.byref(need)))
        ws = torch.full((max(16, need.value) // 4,), float("nan"), device="cuda")
        c.check(L.scr_mlstm_run(c.handle, dtype_code(getattr(torch, dtype)), ctypes.byref(shape), ctypes.byref(st), ptr(pd), p.shape[1], ptr(gd), 2 * H,
                                ptr(bid), ptr(bfd), *[ptr(t) for t in state], ptr(out), ptr(ws), need, stream()))
        o = host(out)
        for f, b in zip(first, who):
            outs[b].append(o[f:f + counts[b]])
            at[b] += counts[b]
        healthy()
    return [np.concatenate(o) for o in outs], state


def plain_memory(m, proj, gates, bi, bf):
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = len(proj)
    p, cap = proj.astype(np.float64), m["gate_cap"]
    q, k, v = p[:, :H * dim].reshape(T, H, dim) * dim ** -0.5, p[:, H * dim:2 * H * dim].reshape(T, H, dim), p[:, 2 * H * dim:2 * H * dim + H * vdim].reshape(T, H, vdim)
    gi = cap * np.tanh((gates[:, :H].astype(np.float64) + bi) / cap)
    gf = plain.log_sigmoid(cap * np.tanh((gates[:, H:].astype(np.float64) + bf) / cap))
    return np.concatenate([plain.mlstm_recurrence(q[:, h], k[:, h], v[:, h], gi[:, h], gf[:, h]) for h in range(H)], 1)


def head_rows(o, H):
    """Each head's readout over its root mean square: what the layer uses (the raw readout may be near a zero of n.q)."""
    return plain.unit_rms(o.reshape(len(o), H, -1), 1e-12)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 24), (1, 32, 32), (3, 48, 72), (2, 128, 256), (1, 256, 64), (2, 10, 13), (1, 144, 40)])
@pytest.mark.parametrize("portions", [[300], [1] * 6 + [2] * 3 + [70] * 5, [64, 64, 1, 63, 8, 9, 200], [7] * 50, [1300], [5, 700, 600]])
def test_recurrence_in_portions(heads, dim, vdim, portions, dtype):
    m = su.memory_spec(heads, dim, vdim, gate_cap=7.0)["mixer"]
    rng = np.random.default_rng(heads * dim + vdim)
    T = sum(portions) if sum(portions) > 1000 else min(sum(portions), 300)
    proj, gates = draw_memory(rng, T, m, dtype), (2.5 * rng.standard_normal((T, 2 * heads))).astype(np.float32)
    bi, bf = rng.standard_normal(heads).astype(np.float32), (2.0 + rng.standard_normal(heads)).astype(np.float32)
    (got,), _ = run_memory(m, dtype, [proj], [gates], bi, bf, [[n] for n in portions], [1])
    want = plain_memory(m, proj, gates, bi, bf)
    tol = 2e-5 if dtype == "float32" else 2e-4                # (the bf16 kernels keep state and weights to about 16 bits)
    err = np.sqrt(((head_rows(got, heads) - head_rows(want, heads)) ** 2).mean(axis=2)).ravel()
    assert np.isfinite(got).all() and np.median(err) < tol / 4
    # a readout whose n.q passes near zero is all cancellation: those few rows only
    assert (err > 4 * tol).mean() < 0.04 and err.max() < 3000 * tol, (np.median(err), np.sort(err)[-5:])


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrence_with_extreme_gates(dtype):
    """Gates at their caps: long memory, instant forgetting, writes far above and far below what is remembered, and the first
    token against the running maximum that starts at zero."""
    H, dim, vdim, T = 4, 32, 40, 200
    m = su.memory_spec(H, dim, vdim, gate_cap=15.0)["mixer"]
    rng = np.random.default_rng(11)
    proj, gates = draw_memory(rng, T, m, dtype), np.zeros((T, 2 * H), np.float32)
    gates[:, 0], gates[:, H] = -40.0, 40.0                       # writes e^-15 below the start, nothing forgotten
    gates[:, 1], gates[:, H + 1] = 40.0, -40.0                   # each token alone
    gates[:, 2], gates[:, H + 2] = np.where(np.arange(T) % 50 == 3, 20.0, -20.0), 6.0      # rare strong writes
    gates[:, 3], gates[:, H + 3] = 0.0, np.where(np.arange(T) % 64 == 0, -40.0, 40.0)      # forgets at chunk starts
    zero = np.zeros(H, np.float32)
    for portions in ([[T]], [[64], [64], [64], [8]], [[1]] * 20 + [[30]] * 6):
        (got,), _ = run_memory(m, dtype, [proj], [gates], zero, zero, portions, [0])
        want = plain_memory(m, proj, gates, zero, zero)
        scale = np.sqrt((want.reshape(T, H, vdim) ** 2).mean(axis=(0, 2)))[None, :, None]
        err = (got - want).reshape(T, H, vdim) / scale
        assert np.sqrt((err ** 2).mean(axis=(0, 2))).max() < (5e-4 if dtype == "float32" else 2e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_of_unequal_sequences_and_of_reused_slots(dtype):
    H, dim, vdim = 2, 32, 48
    m = su.memory_spec(H, dim, vdim)["mixer"]
    rng = np.random.default_rng(5)
    make = lambda T: (draw_memory(rng, T, m, dtype), (2.0 * rng.standard_normal((T, 2 * H))).astype(np.float32))
    seqs = [make(n) for n in (150, 3, 90, 17)]
    long = [make(n) for n in (900, 20, 577, 64)]
    bi, bf = np.zeros(H, np.float32), np.full(H, 2.0, np.float32)
    want = [plain_memory(m, p, g, bi, bf) for p, g in seqs]
    got, state = run_memory(m, dtype, [p for p, _ in seqs], [g for _, g in seqs], bi, bf, [[50, 1, 30, 9], [1, 1, 1, 1], [99, 1, 1, 1], [0, 0, 100, 20]], [3, 0, 2, 1])
    for o, w in zip(got, want):
        assert su.rel(head_rows(o, H), head_rows(w, H)) < (2e-5 if dtype == "float32" else 5e-4)
    # prompts long enough to be cut into groups of chunks, beside short ones, in fresh and then in continued sequences
    got, _ = run_memory(m, dtype, [p for p, _ in long], [g for _, g in long], bi, bf, [[600, 9, 1, 64], [300, 11, 576, 1]], [0, 3, 1, 2], state)
    for o, (p, g) in zip(got, long):
        assert su.rel(head_rows(o, H), head_rows(plain_memory(m, p, g, bi, bf), H)) < (2e-5 if dtype == "float32" else 2e-3)
    p, g = make(20)
    (o,), _ = run_memory(m, dtype, [p], [g], bi, bf, [[9], [11]], [2], state)          # slot 2 again, by a sequence that starts
    assert su.rel(head_rows(o, H), head_rows(plain_memory(m, p, g, bi, bf), H)) < (2e-5 if dtype == "float32" else 5e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_readout_norm_and_gate(dtype):
    from scratchy_b200 import _lib
    from scratchy_b200.dense import dtype_code
    torch = torch_()
    L, c = lib()
    H, vdim, T = 3, 40, 6
    rng = np.random.default_rng(2)
    o, w, g = rng.standard_normal((T, H * vdim)).astype(np.float32), rng.standard_normal(H * vdim).astype(np.float32), draw(rng, (T, H * vdim + 8), dtype)
    o[0] *= 1e-4                                                                     # eps inside the root is at work
    shape = _lib.MlstmShape(H, 16, vdim, 1.0, 1e-5)
    od, wd, gd, y = dev(o), dev(w), dev(g, dtype), torch.empty((T, H * vdim), dtype=getattr(torch, dtype), device="cuda")
    c.check(L.scr_mlstm_finish(c.handle, dtype_code(y.dtype), ctypes.byref(shape), ptr(od), ptr(wd), ptr(gd, 8), g.shape[1], T, ptr(y), stream()))
    want = plain.unit_rms(o.astype(np.float64).reshape(T, H, vdim), 1e-5).reshape(T, -1) * w * plain.sigmoid(g[:, 8:].astype(np.float64))
    assert su.rel(host(y), want) < TOL[dtype] and su.rel(host(y)[0], want[0]) < TOL[dtype]
