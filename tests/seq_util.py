"""Small hybrid-model configurations with random weights for the sequence-model tests, and error measures."""
import json
import os

import numpy as np


def round_bf16(x):
    x = np.ascontiguousarray(x, np.float32)
    b = x.view(np.uint32).astype(np.uint64)
    return ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def attention_spec(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=48, q_rank=56, base=700.0, scale=None, rot_dims=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
        "rot": {"base": base, "dims": rot_dims if rot_dims is not None else rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5}}


def memory_spec(heads=2, dim=16, vdim=24, gate_cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def with_mlp(spec, ff=72, limit=1.5):
    return {**spec, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=88, vocab=210, eps=3e-5, loop=None):
    out = {"architecture": "Vumipel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def random_weights(cfg, seed=0):
    """Every tensor of a configuration, f32 values that bf16 holds exactly."""
    rng = np.random.default_rng(seed)
    W, out = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = round_bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=0.0, std=0.2):
        out[name] = round_bf16(mean + std * rng.standard_normal(n))
    out["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], W)))
    if cfg.get("loop"):
        mat("loop.in", W, 2 * W)
        out["loop.step"] = round_bf16(0.3 * rng.standard_normal((cfg["loop"]["times"], W)))
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W)
        vec(f"l{i}.norm1b", W)
        H = m["heads"]
        if spec["type"] == "latent_attention":
            mat(p + "dq", m["q_rank"], W)
            vec(p + "dq.norm", m["q_rank"], 1.0)
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + "dkv.norm", m["kv_rank"], 1.0)
            mat(p + "uk", H * m["dim"], m["kv_rank"], 1.5)
            mat(p + "uv", H * m["vdim"], m["kv_rank"])
            mat(p + "g", H * m["vdim"], W)
            mat(p + "o", W, H * m["vdim"])
        else:
            for name, n in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * m["vdim"]), ("g", H * m["vdim"])):
                mat(p + name, n, W)
            # keys that lean towards the queries: a readout divided by n.q is a coin toss of sign where n.q is all noise
            out[p + "k"] = round_bf16(0.8 * out[p + "q"] + 0.6 * out[p + "k"])
            mat(p + "i", H, W, 2.0)
            mat(p + "f", H, W, 2.0)
            vec(p + "i.b", H, -1.0, 1.0)
            vec(p + "f.b", H, 3.0, 1.0)
            vec(p + "norm", H * m["vdim"], 1.0)
            mat(p + "o", W, H * m["vdim"])
        if spec.get("mlp") is not None:
            vec(f"l{i}.norm2", W)
            vec(f"l{i}.norm2b", W)
            ff = spec["mlp"]["ff"]
            mat(f"l{i}.mlp.gate", ff, W, 1.5)
            mat(f"l{i}.mlp.up", ff, W, 1.5)
            mat(f"l{i}.mlp.down", W, ff)
    vec("final.norm", W)
    return out


def side_spec(heads=4, kv_heads=2, dim=16, taps=3, bias_max=40, size=24, keep_first=5, scale=None, left_scale=0.7, rheads=3, rdim=16, rvdim=24,
              decay=None, right_scale=1.2, ff=72, weights_of=None):
    """A layer of window attention beside lightning attention."""
    out = {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": taps, "bias_max": bias_max, "scale": scale or dim ** -0.5,
                 "mask": {"size": size, "keep_first": keep_first}},
        "left_scale": left_scale,
        "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay or [float(np.exp(-0.7 * 2.0 ** -i)) for i in range(rheads)]},
        "right_scale": right_scale}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    return out if weights_of is None else {**out, "weights_of": weights_of}


def side_config(layers, width=88, vocab=210, eps=2e-5):
    return {"architecture": "Vekurax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def side_weights(cfg, seed=0, bias_rows=10):
    """Every tensor of a Vekurax configuration, f32 values that bf16 holds exactly."""
    rng = np.random.default_rng(seed)
    W, out = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = round_bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=0.0, std=0.2):
        out[name] = round_bf16(mean + std * rng.standard_normal(n))

    def norm(name, alpha):
        vec(name, W, 1.0)
        vec(name + ".b", W)
        out[name + ".alpha"] = round_bf16(np.array(alpha)).reshape(())
    out["embed"] = round_bf16(rng.standard_normal((cfg["vocab"], W)))
    for i, spec in enumerate(cfg["layers"]):
        if "weights_of" in spec:
            continue
        norm(f"l{i}.norm1", 0.6 + 0.1 * i)
        m, p = spec["mixer"]["left"], f"l{i}.mix.left."
        H, G, dim = m["heads"], m["kv_heads"], m["dim"]
        for name, n in (("q", H * dim), ("k", G * dim)):
            mat(p + name, n, W)
            vec(p + name + ".norm", n, 1.2)
            out[p + name + ".conv"] = round_bf16(0.6 * rng.standard_normal((n, m["conv"])))
            out[p + name + ".conv"][:, -1] = round_bf16(out[p + name + ".conv"][:, -1] + 0.8)
        out[p + "rel"] = round_bf16(rng.standard_normal((bias_rows, H)))
        mat(p + "g", H, W, 2.0)
        mat(p + "o", W, H * dim)
        m, p = spec["mixer"]["right"], f"l{i}.mix.right."
        for name, n in (("q", m["heads"] * m["dim"]), ("k", m["heads"] * m["dim"]), ("v", m["heads"] * m["vdim"]), ("g", m["heads"] * m["vdim"])):
            mat(p + name, n, W, 1.3)
        vec(p + "norm", m["heads"] * m["vdim"], 1.0)
        mat(p + "o", W, m["heads"] * m["vdim"])
        if spec.get("mlp") is not None:
            ff = spec["mlp"]["ff"]
            mat(f"l{i}.mlp.gate", ff, W, 1.5)
            mat(f"l{i}.mlp.up", ff, W, 1.5)
            mat(f"l{i}.mlp.down", W, ff)
    norm("final.norm", 0.5)
    return out


def weights_of(cfg, seed=0):
    return side_weights(cfg, seed) if cfg["architecture"] == "Vekurax" else random_weights(cfg, seed)


def save_checkpoint(directory, cfg, weights):
    from scratchy_b200.weights import write_safetensors
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(directory, "model.safetensors"),
                      {k: ((np.asarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16), "BF16") for k, v in weights.items()})


def make_model(cfg, weights, dtype, **kw):
    """The framework's model on the GPU from host weights."""
    import torch
    from scratchy_b200.layers import GpuWeights
    from scratchy_b200.vekurax import Vekurax, VekuraxConfig
    from scratchy_b200.vumipel import Vumipel, VumipelConfig
    gw = GpuWeights({k: torch.from_numpy(np.asarray(v)).to(torch.bfloat16).cuda() for k, v in weights.items()})
    kw = {"max_tokens": 1024, "max_sequences": 6, **kw}
    if cfg["architecture"] == "Vekurax":
        return Vekurax(VekuraxConfig.from_dict(cfg), gw, "cuda", dtype, **kw)
    return Vumipel(VumipelConfig.from_dict(cfg), gw, "cuda", dtype, **kw)


def tokens_of(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).tolist()


def row_errors(got, want):
    """Per row: rms over the row of the difference (its mean taken off), over the rms of all of `want`."""
    d = np.asarray(got, np.float64) - np.asarray(want, np.float64)
    d -= d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1)) / np.sqrt(np.mean(np.asarray(want, np.float64) ** 2))


def rel(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.linalg.norm(got - want) / max(np.linalg.norm(want), 1e-30))
