"""Plain, slow numpy statement of the sequence models — TEST INFRASTRUCTURE ONLY.

One function per mechanism, float64 throughout, whole sequences from their first token, no cache, no chunks and no
batches: what the framework's kernels, caches and schedules are compared with.  Shares no code with the product.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose stored weight is the difference from one."""
    return unit_rms(x, eps) * (1.0 + w)


def rotate_interleaved(x, positions, dims, base):
    """Rotary positions on the first `dims` of the last axis of x [T, ..., D]; dimension 2i goes with 2i + 1."""
    out = np.array(x, dtype=np.float64)
    for i in range(dims // 2):
        a = positions.astype(np.float64) * base ** (-2.0 * i / dims)
        shape = (len(positions),) + (1,) * (x.ndim - 2)
        c, s = np.cos(a).reshape(shape), np.sin(a).reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_attention(h, w, m, eps):
    """h [T, width]; w: tensors by their short names ('dq', 'dq.norm', ...); m: the mixer's configuration."""
    T = h.shape[0]
    H, dim, rot_dim, vdim, kvr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    cq = unit_rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(T, H, dim + rot_dim)
    dkv = h @ w["dkv"].T
    c = unit_rms(dkv[:, :kvr], eps) * w["dkv.norm"]
    k_rot = rotate_interleaved(dkv[:, kvr:], pos, m["rot"]["dims"], m["rot"]["base"])
    q_rot = rotate_interleaved(q[:, :, dim:], pos, m["rot"]["dims"], m["rot"]["base"])
    k = (c @ w["uk"].T).reshape(T, H, dim)
    v = (c @ w["uv"].T).reshape(T, H, vdim)
    out = np.zeros((T, H, vdim))
    for head in range(H):
        score = (q[:, head, :dim] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        score = np.where(np.tril(np.ones((T, T), bool)), score, -np.inf)
        p = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, head] = (p / p.sum(axis=1, keepdims=True)) @ v[:, head]
    return (out.reshape(T, H * vdim) * sigmoid(h @ w["g"].T)) @ w["o"].T


def mlstm_recurrence(q, k, v, i_log, f_log):
    """One head's matrix memory, token by token.  q, k [T, dim], v [T, vdim], log gates [T] -> o [T, vdim]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    n = np.zeros(k.shape[1])
    mx = 0.0
    out = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        new = max(f_log[t] + mx, i_log[t])
        keep, put = np.exp(f_log[t] + mx - new), np.exp(i_log[t] - new)
        S = keep * S + put * np.outer(k[t], v[t])
        n = keep * n + put * k[t]
        mx = new
        out[t] = (S.T @ q[t]) / (max(abs(n @ q[t]), np.exp(-mx)) + 1e-6)
    return out


def mlstm_gates(h, w, cap):
    i_log = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f_log = log_sigmoid(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    return i_log, f_log


def mlstm(h, w, m, eps):
    T = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vdim)
    i_log, f_log = mlstm_gates(h, w, m["gate_cap"])
    o = np.stack([mlstm_recurrence(q[:, a], k[:, a], v[:, a], i_log[:, a], f_log[:, a]) for a in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(T, H * vdim) * w["norm"]
    return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_mlp(h, w, m):
    return clamped_glu(h @ w["gate"].T, h @ w["up"].T, m["limit"]) @ w["down"].T


def dynamic_tanh(x, alpha, w, b):
    """A norm without statistics: a squashed, scaled and shifted copy of every value."""
    return np.tanh(alpha * x) * w + b


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(u, w):
    """Each channel of u [T, C] with its taps w [C, taps]; the last tap meets the token itself, nothing precedes the first."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def distance_bucket(n, rows, far):
    """Row of a bias table of `rows` rows for a key n tokens back: one row per distance in the first half, the second half
    spaced logarithmically up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(np.floor(np.log(n / half) / np.log(far / half) * (rows - half) + 1e-12)))


def window_visible(T, size, keep_first):
    """[query, key]: the last `size` tokens up to the query itself, and the first `keep_first` of the sequence."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def windowed_softmax(q, k, v, scale, bias, size, keep_first, first=0):
    """One head: queries q at positions first, first + 1, ..., keys k and values v of positions 0, 1, ...; `bias` by distance."""
    T = k.shape[0]
    back = (first + np.arange(q.shape[0]))[:, None] - np.arange(T)[None, :]
    seen = window_visible(T, size, keep_first)[first:first + q.shape[0]]
    score = np.where(seen, q @ k.T * scale + bias[np.maximum(back, 0)], -np.inf)
    p = np.exp(score - score.max(axis=1, keepdims=True))
    return (p / p.sum(axis=1, keepdims=True)) @ v


def window_attention(h, w, m, eps):
    """Grouped heads over a sliding window with kept first tokens.  Queries and keys pass a short convolution and an RMS norm
    over the whole projection; the values are the keys before that norm; a bias per distance and head joins the scores;
    each head's output is gated by one number.  -> [T, width]."""
    T, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(h @ w["q"].T, w["q.conv"])
    k = causal_conv(h @ w["k"].T, w["k.conv"])
    v = k.reshape(T, G, dim)
    q = (unit_rms(q, eps) * w["q.norm"]).reshape(T, H, dim)
    k = (unit_rms(k, eps) * w["k.norm"]).reshape(T, G, dim)
    rows = np.array([distance_bucket(n, w["rel"].shape[0], m["bias_max"]) for n in range(T)])
    out = np.zeros((T, H, dim))
    for head in range(H):
        g = head // (H // G)
        out[:, head] = windowed_softmax(q[:, head], k[:, g], v[:, g], m["scale"], w["rel"][rows, head], m["mask"]["size"], m["mask"]["keep_first"])
    out *= sigmoid(h @ w["g"].T)[:, :, None]
    return out.reshape(T, H * dim) @ w["o"].T


def decayed_memory(q, k, v, decay):
    """One head's matrix memory with a constant decay, token by token.  q, k [T, dim], v [T, vdim] -> o [T, vdim]."""
    S, out = np.zeros((k.shape[1], v.shape[1])), np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def lightning_attention(h, w, m, eps):
    T, H, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ w[n].T).reshape(T, H, dim) for n in ("q", "k"))
    v = silu(h @ w["v"].T).reshape(T, H, vdim)
    o = np.concatenate([decayed_memory(q[:, a], k[:, a], v[:, a], m["decay"][a]) for a in range(H)], axis=1)
    return (unit_rms(o, eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def side_by_side(h, w, m, eps):
    """Two mixers over the same input, their outputs added with a scale each."""
    left = window_attention(h, {k[5:]: v for k, v in w.items() if k.startswith("left.")}, m["left"], eps)
    right = lightning_attention(h, {k[6:]: v for k, v in w.items() if k.startswith("right.")}, m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def gelu_mlp(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def short_names(weights, prefix):
    return {k[len(prefix):]: np.asarray(v, np.float64) for k, v in weights.items() if k.startswith(prefix)}


def layer(x, i, cfg, weights):
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    w = {k: np.asarray(weights[f"l{i}.{k}"], np.float64) for k in ("norm1", "norm2", "norm1b", "norm2b") if f"l{i}.{k}" in weights}
    mixer = MIXERS[spec["type"]]
    y = mixer(norm_around_zero(x, w["norm1"], eps), short_names(weights, f"l{i}.mix."), spec["mixer"], eps)
    x = x + norm_around_zero(y, w["norm1b"], eps)
    if spec.get("mlp") is not None:
        y = dense_mlp(norm_around_zero(x, w["norm2"], eps), short_names(weights, f"l{i}.mlp."), spec["mlp"])
        x = x + norm_around_zero(y, w["norm2b"], eps)
    return x


def vumipel(cfg, weights, tokens):
    """Logits [T, vocab] and the residual stream after every layer run."""
    embed = np.asarray(weights["embed"], np.float64)
    x = embed[np.asarray(tokens)]
    x0 = x.copy()
    runs = []
    loop = cfg.get("loop")
    i = 0
    while i < len(cfg["layers"]):
        if loop and i == loop["start"]:
            w_in, step = np.asarray(weights["loop.in"], np.float64), np.asarray(weights["loop.step"], np.float64)
            for t in range(loop["times"]):
                x = np.concatenate([x, x0], axis=1) @ w_in.T + step[t]
                for j in range(loop["start"], loop["stop"]):
                    x = layer(x, j, cfg, weights)
                    runs.append(x)
            i = loop["stop"]
        else:
            x = layer(x, i, cfg, weights)
            runs.append(x)
            i += 1
    x = norm_around_zero(x, np.asarray(weights["final.norm"], np.float64), cfg["norm"]["eps"])
    return x @ embed.T, runs


def tanh_norm_of(weights, name):
    w, b = (np.asarray(weights[n], np.float64) for n in (name, name + ".b"))
    return lambda x: dynamic_tanh(x, float(weights[name + ".alpha"]), w, b)


def vekurax(cfg, weights, tokens):
    """Logits [T, vocab] and the residual stream after every layer."""
    embed, eps = np.asarray(weights["embed"], np.float64), cfg["norm"]["eps"]
    x, runs = embed[np.asarray(tokens)], []
    for i, spec in enumerate(cfg["layers"]):
        while "weights_of" in cfg["layers"][i]:
            i = cfg["layers"][i]["weights_of"]
        h = tanh_norm_of(weights, f"l{i}.norm1")(x)
        y = side_by_side(h, short_names(weights, f"l{i}.mix."), spec["mixer"], eps)
        if spec.get("mlp") is not None:
            y = y + gelu_mlp(h, short_names(weights, f"l{i}.mlp."))
        x = x + y
        runs.append(x)
    return tanh_norm_of(weights, "final.norm")(x) @ embed.T, runs


def model(cfg, weights, tokens):
    return {"Vumipel": vumipel, "Vekurax": vekurax}[cfg["architecture"]](cfg, weights, tokens)
