"""Every mechanism of side-by-side layers on its own, against the plain statement: joined linears and their ends, dynamic tanh,
short convolutions and whole-projection norms, windowed attention in each of its kernels, the decaying memory token by token
and in chunks."""
import ctypes

import numpy as np
import pytest

from oracle import sequence_plain as plain
from tests import seq_util as su
from tests.test_sequence_ops_gpu import DTYPES, TOL, arena, dev, draw, healthy, host, lib, ptr, stream, torch_

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------ linears
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 7, 16, 17, 50, 200])
@pytest.mark.parametrize("ff,silu,store,f32,K", [(72, 40, 48, 5, 88), (10, 21, 6, 3, 40), (256, 320, 64, 24, 512), (13, 7, 9, 2, 45), (0, 96, 33, 1, 64)])
def test_several_linears_in_one_matrix(M, ff, silu, store, f32, K, dtype):
    from scratchy_b200 import _lib
    from scratchy_b200.dense import JoinedLinear, interleave8
    torch = torch_()
    rng = np.random.default_rng(M + ff + K)
    x = draw(rng, (M, K), dtype)
    mats = {n: draw(rng, (r, K), dtype, 1.5 * K ** -0.5) for n, r in (("gate", ff), ("up", ff), ("silu", silu), ("store", store), ("f32", f32))}
    x64 = x.astype(np.float64)
    out = {n: x64 @ m.astype(np.float64).T for n, m in mats.items()}
    want = {"glu": plain.gelu_tanh(out["gate"]) * out["up"], "silu": plain.silu(out["silu"]), "store": out["store"], "f32": out["f32"]}
    parts = [("silu", dev(mats["silu"], dtype), _lib.PART_SILU), ("store", dev(mats["store"], dtype), _lib.PART_STORE), ("f32", dev(mats["f32"], dtype), _lib.PART_F32)]
    if ff:
        parts.insert(0, ("glu", interleave8(dev(mats["gate"], dtype), dev(mats["up"], dtype)), _lib.PART_GELU_GLU))
    widths = {"glu": (ff + 7) // 8 * 8, "silu": silu, "store": store, "f32": f32}
    bufs = {n: torch.full((M, widths[n] + 8), 7.0, dtype=torch.float32 if n == "f32" else getattr(torch, dtype), device="cuda") for n, _, _ in parts}
    JoinedLinear(parts).run(arena(), dev(x, dtype), {n: b[:, :widths[n]] for n, b in bufs.items()})
    for n, b in bufs.items():
        got, w = host(b), want[n]
        assert su.rel(got[:, :w.shape[1]], w) < (1e-5 if n == "f32" else TOL[dtype]), n
        assert not got[:, w.shape[1]:widths[n]].any() and (got[:, widths[n]:] == 7.0).all(), n
    healthy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 88, 72), (16, 90, 96), (5, 45, 30), (17, 256, 4096), (40, 88, 64), (200, 520, 136), (300, 130, 2048)])
def test_a_linear_that_adds_to_the_residual_and_norms_it(M, N, K, dtype):
    from scratchy_b200.dense import DenseLinear, TanhNorm
    torch = torch_()
    rng = np.random.default_rng(M + N + K)
    x, w, r = draw(rng, (M, K), dtype), draw(rng, (N, K), dtype, K ** -0.5), rng.standard_normal((M, N)).astype(np.float32)
    nw, nb = rng.standard_normal((2, N)).astype(np.float32)
    want = r + x.astype(np.float64) @ w.astype(np.float64).T
    lin, xd = DenseLinear(dev(w, dtype)), dev(x, dtype)
    res = dev(r)
    lin.add_to(arena(), xd, res)
    assert su.rel(host(res), want) < 1e-5
    res, out = dev(r), torch.full((M, N + 8), 7.0, dtype=getattr(torch, dtype), device="cuda")
    lin.add_to(arena(), xd, res, TanhNorm(0.7, dev(nw), dev(nb)), out[:, :N])
    assert su.rel(host(res), want) < 1e-5
    assert su.rel(host(out)[:, :N], plain.dynamic_tanh(want, 0.7, nw, nb)) < TOL[dtype] and (host(out)[:, N:] == 7.0).all()
    healthy()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [88, 45, 3072])
def test_dynamic_tanh_of_all_and_of_chosen_rows(W, dtype):
    from scratchy_b200.dense import TanhNorm, seq_norm
    torch = torch_()
    rng = np.random.default_rng(W)
    x = (3.0 * rng.standard_normal((9, W))).astype(np.float32)
    w, b = rng.standard_normal((2, W)).astype(np.float32)
    norm = TanhNorm(0.35, dev(w), dev(b))
    want = plain.dynamic_tanh(x.astype(np.float64), 0.35, w, b)
    xd, out = dev(x), torch.empty((9, W), dtype=getattr(torch, dtype), device="cuda")
    seq_norm(xd, 1e-5, out=out, tanh=norm)
    assert su.rel(host(out), want) < TOL[dtype] and (host(xd) == x).all()
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device="cuda")
    out = torch.empty((3, W), dtype=getattr(torch, dtype), device="cuda")
    seq_norm(xd, 1e-5, out=out, tanh=norm, row_index=rows)
    assert su.rel(host(out), want[[7, 0, 3]]) < TOL[dtype]
    healthy()


# ------------------------------------------------------------------------------------------------ windowed attention
LN2 = float(np.log(2.0))


class Window:
    """Sequences of a window attention over randomly placed blocks: drawn projections or drawn queries and values."""
    BLOCK = 64

    def __init__(self, heads, kv_heads, dim, window, keep_first, n_bias, lengths, dtype, seed=0, taps=3, scale=None, eps=1e-5):
        self.H, self.G, self.dim, self.window, self.keep, self.n_bias, self.dtype, self.taps = heads, kv_heads, dim, window, keep_first, n_bias, dtype, taps
        self.scale, self.eps, self.lengths = scale or dim ** -0.5, eps, lengths
        self.rng = np.random.default_rng(seed)
        self.max_blocks = max(-(-n // self.BLOCK) for n in lengths)
        self.num_blocks = self.max_blocks * len(lengths) + 3
        order = self.rng.permutation(self.num_blocks)
        self.blocks = [order[b * self.max_blocks:(b + 1) * self.max_blocks] for b in range(len(lengths))]
        torch = torch_()
        self.cache = torch.full((self.num_blocks * self.BLOCK, kv_heads * dim), 3.0, dtype=getattr(torch, dtype), device="cuda")
        self.key_scale = torch.full((self.num_blocks * self.BLOCK,), 5.0, device="cuda")
        self.bias = self.rng.standard_normal((heads, n_bias)).astype(np.float32)

    def rows_of(self, b, n):
        p = np.arange(n)
        return torch_().from_numpy(self.blocks[b][p // self.BLOCK] * self.BLOCK + p % self.BLOCK).cuda()

    def shape(self, out_scale=1.0):
        from scratchy_b200 import _lib
        return _lib.WindowShape(self.H, self.G, self.dim, self.taps, self.window, self.keep, self.n_bias, self.BLOCK, self.num_blocks, self.max_blocks, self.eps,
                                self.scale, out_scale)

    def step(self, counts, starts, slots=None, hide_unseen=False):
        """Device description of a step of `counts` rows of every sequence from positions `starts`."""
        from scratchy_b200 import _lib
        torch = torch_()
        seg, pos, segs, row = [], [], [], 0
        table = np.stack(self.blocks).astype(np.int32)
        for b, (n, p) in enumerate(zip(counts, starts)):
            seg += [b] * n
            pos += range(p, p + n)
            segs.append([row, n, p, slots[b] if slots else b])
            row += n
            if hide_unseen:                                   # blocks that no row sees are not in the table
                for k in range(self.max_blocks):
                    lo, hi = k * self.BLOCK, (k + 1) * self.BLOCK
                    if (hi <= p - self.window + 1 and lo >= self.keep) or lo >= p + n:
                        table[b, k] = -1
        self.kept = [torch.from_numpy(np.array(a, np.int32)).cuda() for a in (seg, pos, segs)] + [torch.from_numpy(table).cuda()]
        return _lib.Step(*(t.data_ptr() for t in self.kept), row, len(counts), max(counts), max(p + n for n, p in zip(counts, starts)), 1 + (max(slots) if slots else len(counts)))

    def padded_bias(self):
        from scratchy_b200 import _lib
        b = self.bias / LN2
        return dev(np.concatenate([np.repeat(b[:, :1], _lib.BIAS_LO, 1), b, np.repeat(b[:, -1:], _lib.BIAS_HI, 1)], 1))

    def attend(self, q, gate, counts, starts, out_scale=1.0, **kw):
        """q [rows, heads * dim] against what the cache holds -> [rows, heads, dim]."""
        from scratchy_b200.dense import dtype_code
        torch = torch_()
        L, c = lib()
        st, sh = self.step(counts, starts, **kw), self.shape(out_scale)
        qd, gd, bd = dev(q, self.dtype), dev(gate), self.padded_bias()
        out = torch.full((len(q), self.H * self.dim + 8), 7.0, dtype=qd.dtype, device="cuda")
        c.check(L.scr_window_attention(c.handle, dtype_code(qd.dtype), ctypes.byref(sh), ctypes.byref(st), ptr(qd), ptr(self.cache), ptr(self.key_scale), ptr(bd), ptr(gd),
                                       gate.shape[1], ptr(out), out.shape[1], stream()))
        healthy()
        got = host(out)
        assert (got[:, self.H * self.dim:] == 7.0).all()
        return got[:, :self.H * self.dim].reshape(len(q), self.H, self.dim)

    def fill(self, values, inverse):
        """values[b] [length, kv_heads, dim]; inverse[b] [length]: reciprocal root mean squares."""
        torch = torch_()
        for b, (v, i) in enumerate(zip(values, inverse)):
            self.cache[self.rows_of(b, len(v))] = dev(v.reshape(len(v), -1), self.dtype)
            self.key_scale[self.rows_of(b, len(v))] = dev(i * self.scale / LN2)

    def plain(self, b, q, values, inverse, gate, first, out_scale=1.0):
        n, out = len(q), np.zeros((len(q), self.H, self.dim))
        bias = lambda h: np.concatenate([self.bias[h], np.repeat(self.bias[h, -1:], max(0, first + n - self.n_bias))]).astype(np.float64)
        for h in range(self.H):
            g = h // (self.H // self.G)
            v = values[b][:first + n, g].astype(np.float64)
            k = v * inverse[b][:first + n, None]
            out[:, h] = plain.windowed_softmax(q[:, h].astype(np.float64), k, v, self.scale, bias(h), self.window, self.keep, first)
        return out * plain.sigmoid(gate.astype(np.float64))[:, :, None] * out_scale


SHAPES = [(4, 2, 16), (3, 1, 64), (6, 6, 128), (8, 2, 40), (12, 1, 32), (2, 1, 256), (5, 1, 10), (2, 2, 96)]
STEPS = [((1, 1, 1), (0, 70, 299)), ((5, 2, 30), (0, 63, 200)), ((64, 1, 129), (0, 300, 130)), ((300, 90, 3), (0, 201, 7)), ((257, 128, 64), (43, 65, 64))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim", SHAPES)
@pytest.mark.parametrize("counts,starts", STEPS)
@pytest.mark.parametrize("window,keep_first,n_bias", [(70, 5, 40), (1000, 0, 1), (1, 0, 3), (64, 64, 90), (33, 130, 400)])
def test_window_attention_over_the_paged_cache(heads, kv_heads, dim, counts, starts, window, keep_first, n_bias, dtype):
    lengths = [n + p for n, p in zip(counts, starts)]
    w = Window(heads, kv_heads, dim, window, keep_first, n_bias, lengths, dtype, seed=heads * dim + window)
    v = [draw(w.rng, (n, kv_heads, dim), dtype) for n in lengths]
    inv = [(0.5 + w.rng.random(n)).astype(np.float32) for n in lengths]
    w.fill(v, inv)
    q, gate = draw(w.rng, (sum(counts), heads, dim), dtype), w.rng.standard_normal((sum(counts), heads)).astype(np.float32)
    got = w.attend(q.reshape(len(q), -1), gate, counts, starts, out_scale=0.6, hide_unseen=True)
    row = 0
    for b, (n, p) in enumerate(zip(counts, starts)):
        want = w.plain(b, q[row:row + n], v, inv, gate[row:row + n], p, 0.6)
        assert su.rel(got[row:row + n], want) < TOL[dtype], b
        row += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 64), (3, 1, 128), (2, 1, 24)])
def test_one_key_that_stands_out_at_every_edge(heads, kv_heads, dim, dtype):
    """A key far above all others, just inside and just outside the window, the kept first tokens and the blocks: the output is its
    value exactly where it is visible, in a prompt and for a single token."""
    window, keep, T = 150, 70, 520
    w = Window(heads, kv_heads, dim, window, keep, 30, [T], dtype, seed=9)
    base = draw(w.rng, (T, kv_heads, dim), dtype, 0.05)
    q, gate = np.zeros((T, heads, dim), np.float32), np.full((T, heads), 20.0, np.float32)
    q[:, :, 0] = 8.0
    inv = [np.ones(T, np.float32)]
    for at in (0, 63, 64, 69, 70, 71, 127, 128, 255, 369, 370, 371):
        v = [base.copy()]
        v[0][at, :, 0] = 16.0 * dim ** 0.5
        w.fill(v, inv)
        want = w.plain(0, q, v, inv, gate, 0)
        seen = plain.window_visible(T, window, keep)[:, at]
        strong = want[:, :, 0] > 4.0 * dim ** 0.5
        assert (strong == seen[:, None]).all()
        assert su.rel(w.attend(q.reshape(T, -1), gate, [T], [0]), want) < TOL[dtype]
        for p in sorted({at, min(at + window - 1, T - 1), min(at + window, T - 1), T - 1}):
            got = w.attend(q[p:p + 1].reshape(1, -1), gate[:1], [1], [p], hide_unseen=True)
            assert su.rel(got, want[p:p + 1]) < 2 * TOL[dtype], (at, p)
            if p + 3 <= T:
                assert su.rel(w.attend(q[p:p + 3].reshape(3, -1), gate[:3], [3], [p], hide_unseen=True), want[p:p + 3]) < 2 * TOL[dtype], (at, p)


@pytest.mark.parametrize("dtype", DTYPES)
def test_scores_that_climb_along_the_sequence_rescale_the_sums(dtype):
    T, H = 600, 2
    w = Window(H, 1, 64, 400, 3, 1, [T], dtype, seed=3, scale=1.0)
    v = [draw(w.rng, (T, 1, 64), dtype)]
    v[0][:, 0, 0] = su.round_bf16(np.linspace(-4.0, 4.0, T))
    inv = [np.ones(T, np.float32)]
    w.fill(v, inv)
    q, gate = draw(w.rng, (T, H, 64), dtype, 0.1), np.zeros((T, H), np.float32)
    q[:, 0, 0], q[:, 1, 0] = 15.0, -15.0
    assert su.rel(w.attend(q.reshape(T, -1), gate, [T], [0]), w.plain(0, q, v, inv, gate, 0)) < TOL[dtype]
    for p in (0, 1, 399, 400, 403, 599):
        assert su.rel(w.attend(q[p:p + 1].reshape(1, -1), gate[:1], [1], [p]), w.plain(0, q[p:p + 1], v, inv, gate[:1], p)) < 2 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,taps", [(4, 2, 16, 3), (2, 1, 64, 4), (3, 3, 40, 1), (6, 2, 24, 2), (3, 1, 10, 3), (2, 2, 16, 6), (40, 8, 128, 4), (70, 2, 128, 3)])
@pytest.mark.parametrize("portions", [[60], [1] * 8 + [2, 3, 1, 20, 1, 25], [5, 1, 1, 40, 13], [2] * 30])
def test_convolution_norm_and_cache_append_in_portions(heads, kv_heads, dim, taps, portions, dtype):
    """Two sequences side by side, the second one token ahead in its cut, on slots that held something before."""
    from scratchy_b200.dense import dtype_code
    torch = torch_()
    T = sum(portions)
    w = Window(heads, kv_heads, dim, 100, 0, 4, [T, T], dtype, seed=taps + dim, taps=taps)
    L, c = lib()
    C, nq = (heads + kv_heads) * dim, heads * dim
    proj = [draw(w.rng, (T, C), dtype) for _ in range(2)]
    conv, wq, wk = w.rng.standard_normal((C, taps)).astype(np.float32), (1 + 0.3 * w.rng.standard_normal(nq)).astype(np.float32), (1 + 0.3 * w.rng.standard_normal(C - nq)).astype(np.float32)
    folded = wq * np.repeat(wk.reshape(kv_heads, 1, dim), heads // kv_heads, 1).reshape(-1)
    conv_d, norm_d = dev(conv.T), dev(folded)
    state = torch.full((3, max(1, taps - 1), C), float("nan"), dtype=w.cache.dtype, device="cuda")
    queries = [[], []]
    second = [1] + portions
    at = [0, 0]
    for a, b in zip(portions + [0], second):
        counts = [a, min(b, T - at[1])]
        who = [i for i in range(2) if counts[i]]
        if not who:
            continue
        st = w.step([counts[i] for i in who], [at[i] for i in who], slots=[(2, 0)[i] for i in who])
        w.kept[3] = torch.from_numpy(np.stack([w.blocks[i] for i in who]).astype(np.int32)).cuda()
        st.block_table, st.num_slots = w.kept[3].data_ptr(), 3
        rows = np.concatenate([proj[i][at[i]:at[i] + counts[i]] for i in who])
        padded = dev(np.concatenate([rows, np.zeros((len(rows), 8), np.float32)], 1), dtype)
        q = torch.full((len(rows), nq), float("nan"), dtype=w.cache.dtype, device="cuda")
        c.check(L.scr_window_prepare(c.handle, dtype_code(q.dtype), ctypes.byref(w.shape()), ctypes.byref(st), ptr(padded), C + 8, ptr(conv_d), ptr(norm_d), ptr(state), ptr(q),
                                     ptr(w.cache), ptr(w.key_scale), stream()))
        healthy()
        r = 0
        for i in who:
            queries[i].append(host(q)[r:r + counts[i]])
            r += counts[i]
            at[i] += counts[i]
    assert at == [T, T]
    for i in range(2):
        y = plain.causal_conv(proj[i].astype(np.float64), conv.astype(np.float64))
        want_q = plain.unit_rms(y[:, :nq], w.eps) * folded
        assert su.rel(np.concatenate(queries[i]), want_q) < TOL[dtype]
        rows = w.rows_of(i, T)
        assert su.rel(host(w.cache[rows]), y[:, nq:]) < TOL[dtype]
        inv = 1.0 / np.sqrt(np.mean(y[:, nq:] ** 2, axis=1) + w.eps)
        assert su.rel(host(w.key_scale[rows]), inv * w.scale / LN2) < 1e-5
        if taps > 1:
            past = np.concatenate([np.zeros((taps - 1, C)), proj[i]])[-(taps - 1):]
            assert (host(state[(2, 0)[i]]) == past).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("counts", [[500, 1, 1, 2, 1, 3, 90], [1] * 320, [700], [296, 5]])
def test_convolution_over_many_rows_of_many_sequences(counts, dtype):
    from scratchy_b200.dense import dtype_code
    torch = torch_()
    heads, kv_heads, dim, taps = 4, 2, 32, 4
    starts = [(7 * i) % 5 for i in range(len(counts))]           # some start afresh, some with one to four tokens behind them
    w = Window(heads, kv_heads, dim, 100, 0, 4, [n + p for n, p in zip(counts, starts)], dtype, seed=len(counts), taps=taps)
    L, c = lib()
    C, nq, B = (heads + kv_heads) * dim, heads * dim, len(counts)
    full = [draw(w.rng, (n + p, C), dtype) for n, p in zip(counts, starts)]
    conv, norm = w.rng.standard_normal((C, taps)).astype(np.float32), (1 + 0.3 * w.rng.standard_normal(nq)).astype(np.float32)
    past = np.stack([np.concatenate([np.full((taps - 1, C), 9.0), f[:p]])[-(taps - 1):] for f, p in zip(full, starts)])
    state, rows = dev(past, dtype), np.concatenate([f[p:] for f, p in zip(full, starts)])
    st = w.step(counts, starts)
    q = torch.full((len(rows), nq), float("nan"), dtype=w.cache.dtype, device="cuda")
    rd, conv_d, norm_d = dev(rows, dtype), dev(conv.T), dev(norm)
    c.check(L.scr_window_prepare(c.handle, dtype_code(q.dtype), ctypes.byref(w.shape()), ctypes.byref(st), ptr(rd), C, ptr(conv_d), ptr(norm_d), ptr(state), ptr(q), ptr(w.cache),
                                 ptr(w.key_scale), stream()))
    healthy()
    got, r = host(q), 0
    for b, (f, n, p) in enumerate(zip(full, counts, starts)):
        y = plain.causal_conv(f.astype(np.float64), conv.astype(np.float64))[p:]
        assert su.rel(got[r:r + n], plain.unit_rms(y[:, :nq], w.eps) * norm) < TOL[dtype], b
        at = w.rows_of(b, n + p)[p:]
        assert su.rel(host(w.cache[at]), y[:, nq:]) < TOL[dtype], b
        assert su.rel(host(w.key_scale[at]), w.scale / LN2 / np.sqrt(np.mean(y[:, nq:] ** 2, axis=1) + w.eps)) < 1e-5, b
        assert (host(state[b]) == np.concatenate([np.zeros((taps - 1, C)), f])[-(taps - 1):]).all(), b
        r += n


# ------------------------------------------------------------------------------------------------ decaying memory
def run_lightning(m, dtype, proj, portions, slots, state=None):
    """Runs the rows of each sequence in the given portions; returns readouts per sequence and the state."""
    from scratchy_b200 import _lib
    from scratchy_b200.dense import dtype_code
    from scratchy_b200.mixers import decay_powers
    torch = torch_()
    L, c = lib()
    H, dim, vdim, B = m["heads"], m["dim"], m["vdim"], len(proj)
    shape, total = _lib.LightningShape(H, dim, vdim, 1e-5, 1.0), max(slots) + 1
    powers = decay_powers(np.asarray(m["decay"], np.float64)).cuda()
    state = torch.full((total, H, dim, vdim), float("nan"), device="cuda") if state is None else state          # a fresh sequence ignores what the slot holds
    outs, at = [[] for _ in range(B)], [0] * B
    for step in portions:
        counts = [min(n, len(proj[b]) - at[b]) for b, n in enumerate(step)]
        who = [b for b in range(B) if counts[b] > 0]
        if not who:
            break
        p = np.concatenate([proj[b][at[b]:at[b] + counts[b]] for b in who])
        first = np.cumsum([0] + [counts[b] for b in who])[:-1]
        segs = torch.from_numpy(np.array([[f, counts[b], at[b], slots[b]] for f, b in zip(first, who)], np.int32)).cuda()
        st = _lib.Step(0, 0, segs.data_ptr(), 0, len(p), len(who), max(counts), 0, total)
        pd, out = dev(p, dtype), torch.full((len(p), H * vdim), float("nan"), device="cuda")
        need = ctypes.c_size_t(0)
        c.check(L.scr_lightning_workspace(dtype_code(pd.dtype), ctypes.byref(shape), ctypes.byref(st), ctypes.byref(need)))
        ws = torch.full((max(16, need.value) // 4,), float("nan"), device="cuda")
        c.check(L.scr_lightning_run(c.handle, dtype_code(pd.dtype), ctypes.byref(shape), ctypes.byref(st), ptr(pd), p.shape[1], ptr(powers), ptr(state), ptr(out), ptr(ws), need,
                                    stream()))
        o = host(out)
        for f, b in zip(first, who):
            outs[b].append(o[f:f + counts[b]])
            at[b] += counts[b]
        healthy()
    return [np.concatenate(o) for o in outs], state


def plain_lightning(m, proj):
    H, dim, vdim, T = m["heads"], m["dim"], m["vdim"], len(proj)
    p = proj.astype(np.float64)
    q, k, v = p[:, :H * dim].reshape(T, H, dim), p[:, H * dim:2 * H * dim].reshape(T, H, dim), p[:, 2 * H * dim:].reshape(T, H, vdim)
    return np.concatenate([plain.decayed_memory(q[:, h], k[:, h], v[:, h], m["decay"][h]) for h in range(H)], 1)


def per_head(got, want, H):
    """Worst head's relative error (a head that remembers long outweighs the others)."""
    g, w = got.reshape(len(got), H, -1), want.reshape(len(want), H, -1)
    return max(su.rel(g[:, h], w[:, h]) for h in range(H))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 24), (1, 32, 32), (3, 48, 72), (2, 128, 256), (1, 256, 64), (2, 10, 13), (1, 144, 40), (2, 7, 6), (1, 300, 20)])
@pytest.mark.parametrize("portions", [[300], [1] * 6 + [2] * 3 + [70] * 5, [64, 64, 1, 63, 8, 9, 200], [7] * 50, [1300], [5, 700, 600]])
def test_decaying_memory_in_portions(heads, dim, vdim, portions, dtype):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": [0.999, 0.6, 0.97][:heads]}
    rng = np.random.default_rng(heads * dim + vdim)
    T = sum(portions) if sum(portions) > 1000 else min(sum(portions), 300)
    proj = draw(rng, (T, heads * (2 * dim + vdim)), dtype)
    (got,), _ = run_lightning(m, dtype, [proj], [[n] for n in portions], [1])
    assert np.isfinite(got).all() and per_head(got, plain_lightning(m, proj), heads) < (4e-6 if dtype == "float32" else 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_at_their_limits(dtype):
    m = {"heads": 4, "dim": 32, "vdim": 40, "decay": [0.0, 1.0, 1e-6, 0.99999]}
    proj = draw(np.random.default_rng(1), (400, 4 * 104), dtype)
    for portions in ([[400]], [[64], [64], [72]], [[1]] * 20 + [[30]] * 20):
        (got,), _ = run_lightning(m, dtype, [proj], portions, [0])
        assert per_head(got, plain_lightning(m, proj[:len(got)]), 4) < (4e-6 if dtype == "float32" else 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_memories_of_unequal_sequences_and_of_reused_slots(dtype):
    m = {"heads": 2, "dim": 32, "vdim": 48, "decay": [0.995, 0.8]}
    rng = np.random.default_rng(5)
    make = lambda T: draw(rng, (T, 2 * 112), dtype)
    tol = 4e-6 if dtype == "float32" else 1e-4
    seqs, long = [make(n) for n in (150, 3, 90, 17)], [make(n) for n in (900, 20, 577, 64)]
    got, state = run_lightning(m, dtype, seqs, [[50, 1, 30, 9], [1, 1, 1, 1], [99, 1, 1, 1], [0, 0, 100, 20]], [3, 0, 2, 1])
    assert all(per_head(o, plain_lightning(m, p), 2) < tol for o, p in zip(got, seqs))
    got, _ = run_lightning(m, dtype, long, [[600, 9, 1, 64], [300, 11, 576, 1]], [0, 3, 1, 2], state)
    assert all(per_head(o, plain_lightning(m, p), 2) < tol for o, p in zip(got, long))
    p = make(20)
    (o,), _ = run_lightning(m, dtype, [p], [[9], [11]], [2], state)                  # slot 2 again, by a sequence that starts
    assert per_head(o, plain_lightning(m, p), 2) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,vdim", [(3, 40), (12, 256), (3, 13), (5, 1000), (40, 256)])
def test_readout_norm_over_all_heads_and_gate(H, vdim, dtype):
    from scratchy_b200 import _lib
    from scratchy_b200.dense import dtype_code
    torch = torch_()
    L, c = lib()
    n, T = H * vdim, 6
    rng = np.random.default_rng(n)
    o, w, g = rng.standard_normal((T, n)).astype(np.float32), rng.standard_normal(n).astype(np.float32), draw(rng, (T, n + 8), dtype)
    o[0] *= 1e-3                                                                     # eps inside the root is at work
    shape = _lib.LightningShape(H, 16, vdim, 1e-5, -0.8)
    od, wd, gd, y = dev(o), dev(w), dev(g, dtype), torch.full((T, n + 16), 7.0, dtype=getattr(torch, dtype), device="cuda")
    c.check(L.scr_lightning_finish(c.handle, dtype_code(y.dtype), ctypes.byref(shape), ptr(od), ptr(wd), ptr(gd, 8), g.shape[1], T, ptr(y), y.shape[1], stream()))
    want = plain.unit_rms(o.astype(np.float64), 1e-5) * w * plain.sigmoid(g[:, 8:].astype(np.float64)) * -0.8
    assert su.rel(host(y)[:, :n], want) < TOL[dtype] and su.rel(host(y)[0, :n], want[0]) < TOL[dtype] and (host(y)[:, n:] == 7.0).all()
    healthy()
