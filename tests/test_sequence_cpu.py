"""Sequence models, host side: the plain statement against hand-computed cases, configuration, bookkeeping, scheduling and
trace replay on a model that only records what it is asked to run."""
import io
import json
import types

import numpy as np
import pytest

from oracle import sequence_plain as plain
from scratchy_b200 import registry, trace
from scratchy_b200.engine import Engine
from scratchy_b200.sequences import OutOfCache, SequenceTable
from tests import seq_util as su


# ---------------------------------------------------------------------------------------- the plain statement
def test_norm_keeps_eps_inside_the_root():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(plain.unit_rms(x, 0.0), x / np.sqrt(12.5))
    assert np.allclose(plain.norm_around_zero(np.zeros((1, 4)), np.ones(4), 1e-5), 0.0)
    assert np.allclose(plain.norm_around_zero(x, np.array([1.0, -0.5]), 2.0), x / np.sqrt(14.5) * np.array([2.0, 0.5]))


def test_rotation_pairs_neighbours_and_leaves_the_rest():
    x = np.array([[1.0, 0.0, 0.0, 1.0, 5.0, 6.0]])
    out = plain.rotate_interleaved(x, np.array([2]), 4, 100.0)
    a, b = 2.0, 2.0 * 100.0 ** -0.5
    assert np.allclose(out, [[np.cos(a), np.sin(a), -np.sin(b), np.cos(b), 5.0, 6.0]])


def test_recurrence_of_one_token_and_of_a_forgotten_past():
    q, k, v = np.array([[2.0, 0.0]]), np.array([[0.5, 1.0]]), np.array([[3.0, -1.0, 4.0]])
    o = plain.mlstm_recurrence(q, k, v, np.array([0.7]), np.array([-0.1]))
    # m = max(-0.1, 0.7) = 0.7, S = k v^T, n = k, n.q = 1 against e^-0.7
    assert np.allclose(o, v * 1.0 / (1.0 + 1e-6))
    # an input gate far below the running maximum writes e^(i - m)
    o = plain.mlstm_recurrence(q, k, v, np.array([-5.0]), np.array([-0.5]))
    m, w = -0.5, np.exp(-4.5)
    assert np.allclose(o, v * w / (max(w, np.exp(-m)) + 1e-6))
    # a closed forget gate in between leaves only the later token
    q2, k2, v2 = np.repeat(q, 2, 0), np.array([[9.0, 9.0], [0.5, 1.0]]), np.array([[7.0, 7.0, 7.0], [3.0, -1.0, 4.0]])
    o = plain.mlstm_recurrence(q2, k2, v2, np.array([0.0, 0.0]), np.array([0.0, -60.0]))
    assert np.allclose(o[1], v2[1] / (1.0 + 1e-6))


def test_clamped_unit_clamps_each_side_its_own_way():
    g, u = np.array([5.0, -5.0, 1.0]), np.array([4.0, -4.0, 0.5])
    a, b = np.array([2.0, -5.0, 1.0]), np.array([2.0, -2.0, 0.5])
    assert np.allclose(plain.clamped_glu(g, u, 2.0), a / (1.0 + np.exp(-1.702 * a)) * (b + 1.0))


def test_attention_of_the_first_token_is_its_own_value():
    spec = su.attention_spec()["mixer"]
    w = {k[7:]: v for k, v in su.random_weights(su.config([su.with_mlp(su.attention_spec(), None)])).items() if k.startswith("l0.mix.")}
    h = np.random.default_rng(0).standard_normal((3, 88))
    out = plain.latent_attention(h, w, spec, 1e-5)
    c = plain.unit_rms((h[:1] @ w["dkv"].T)[:, :48], 1e-5) * w["dkv.norm"]
    want = ((c @ w["uv"].T) / (1.0 + np.exp(-(h[:1] @ w["g"].T)))) @ w["o"].T
    assert np.allclose(out[:1], want)


def test_dynamic_tanh_and_gelu():
    x = np.array([[0.0, 2.0, -1.0]])
    assert np.allclose(plain.dynamic_tanh(x, 0.5, np.array([1.0, 2.0, 3.0]), np.array([0.1, 0.2, 0.3])), [[0.1, 2 * np.tanh(1.0) + 0.2, 3 * np.tanh(-0.5) + 0.3]])
    assert np.allclose(plain.gelu_tanh(np.array([0.0, 1.0, -1.0, 10.0])), [0.0, 0.841192, -0.158808, 10.0], atol=1e-6)


def test_convolution_ends_with_the_token_itself():
    u = np.array([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]])
    w = np.array([[0.5, 0.0, 1.0], [0.0, 2.0, 0.0]])
    assert np.allclose(plain.causal_conv(u, w), [[1.0, 0.0], [2.0, 20.0], [3.5, 40.0]])


def test_buckets_of_key_distances():
    from scratchy_b200.mixers import distance_bias, distance_buckets
    assert distance_buckets(8, 64)[:5] == [0, 1, 2, 3, 4]
    assert [plain.distance_bucket(n, 8, 64) for n in (4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    for rows, far in ((8, 64), (16, 100), (32, 128), (7, 50), (2, 9), (6, 4), (10, 160), (24, 3000)):
        t = distance_buckets(rows, far)
        assert t[-1] == rows - 1 and all(a <= b for a, b in zip(t, t[1:])) and (len(t) == 1 or t[-2] < rows - 1)
        assert all(t[min(n, len(t) - 1)] == plain.distance_bucket(n, rows, far) for n in range(0, 4000, 1 if far < 500 else 7))
    assert distance_buckets(1, 20) == [0]
    import torch
    from scratchy_b200 import _lib
    rel = torch.arange(16.0).reshape(8, 2)
    bias, n = distance_bias(rel, 64)
    assert n == 33 and bias.shape == (2, _lib.BIAS_LO + n + _lib.BIAS_HI)
    assert torch.allclose(bias[1, _lib.BIAS_LO + 16] * np.log(2.0), rel[6, 1]) and torch.equal(bias[:, 0], bias[:, _lib.BIAS_LO]) and torch.equal(bias[:, -1], bias[:, _lib.BIAS_LO + n - 1])


def test_windows_keep_the_first_tokens():
    seen = plain.window_visible(7, 3, 2)
    assert [seen[6].tolist(), seen[3].tolist(), seen[1].tolist()] == [[1, 1, 0, 0, 1, 1, 1], [1, 1, 1, 1, 0, 0, 0], [1, 1, 0, 0, 0, 0, 0]]
    v = np.arange(7.0)[:, None]
    out = plain.windowed_softmax(np.zeros((1, 1)), v, v, 1.0, np.zeros(7), 3, 2, first=6)
    assert np.allclose(out, (0 + 1 + 4 + 5 + 6) / 5)
    bias = np.array([0.0, 0, 0, 0, 0, 50.0, 0])                                # a distance of 5 stands out: key 1
    assert np.allclose(plain.windowed_softmax(np.zeros((1, 1)), v, v, 1.0, bias, 3, 2, first=6), 1.0)


def test_decayed_memory_forgets_at_its_rate():
    q, k, v = np.ones((3, 1)), np.array([[1.0], [0.0], [2.0]]), np.array([[1.0, 4.0], [9.0, 9.0], [1.0, 0.0]])
    assert np.allclose(plain.decayed_memory(q, k, v, 0.5), [[1.0, 4.0], [0.5, 2.0], [2.25, 1.0]])


# ---------------------------------------------------------------------------------------- configuration and registry
def test_runs_of_a_loop():
    from scratchy_b200.vumipel import VumipelConfig
    layers = [su.with_mlp(su.memory_spec()) for _ in range(4)]
    runs = lambda loop: VumipelConfig.from_dict(su.config(layers, loop=loop)).runs()
    assert runs(None) == [(0, None), (1, None), (2, None), (3, None)]
    assert runs((1, 3, 2)) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert runs((0, 1, 3)) == [(0, 0), (0, 1), (0, 2), (1, None), (2, None), (3, None)]
    assert runs((3, 4, 1)) == [(0, None), (1, None), (2, None), (3, 0)]
    for bad in ((2, 2, 1), (0, 5, 1), (0, 1, 0)):
        with pytest.raises(ValueError):
            runs(bad)


def test_layers_on_the_weights_of_earlier_ones():
    from scratchy_b200.vekurax import VekuraxConfig
    S = su.side_spec
    cfg = VekuraxConfig.from_dict(su.side_config([S(size=9, keep_first=4), S(), S(weights_of=0), S(weights_of=2), S(weights_of=1)]))
    assert cfg.owners() == [0, 1, 0, 0, 1] and (cfg.window, cfg.keep_first) == (24, 5)
    for bad in (1, 2, -1):
        with pytest.raises(ValueError):
            VekuraxConfig.from_dict(su.side_config([S(), S(weights_of=bad)]))
    with pytest.raises(ValueError, match="serial"):
        VekuraxConfig.from_dict(su.side_config([{**S(), "type": "serial"}]))


def test_every_design_has_the_kernels_it_needs_and_no_others():
    from scratchy_b200 import build
    assert set(build.DESIGNS) == set(registry.ARCHITECTURES) - {"LlamaForCausalLM"}
    vek = set(build.LIBRARIES[build.design_path("Vekurax")])
    assert set(build.MODELS_COMMON) < vek and "window_prefill.cu" in vek and not any(s.startswith(("latent", "mlstm", "fp8", "affine")) for s in vek)
    assert vek < set(build.MODELS_SOURCES)


def test_unknown_mixer_and_architecture_are_refused():
    from scratchy_b200.vumipel import VumipelConfig
    cfg = su.config([{"type": "convolution", "mixer": {}, "mlp": None}])
    with pytest.raises(ValueError, match="convolution"):
        VumipelConfig.from_dict(cfg)
    with pytest.raises(ValueError, match="Nobody"):
        registry.architecture_of({"architecture": "Nobody"})
    assert registry.architecture_of({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    assert registry.model_class(su.config([])).__name__ == "Vumipel"
    assert registry.model_class(su.side_config([])).__name__ == "Vekurax"


def test_llama_configuration_from_a_checkpoint_folder():
    from scratchy_b200.llama_serving import config_from_dict
    c = config_from_dict({"hidden_size": 512, "num_hidden_layers": 2, "num_attention_heads": 4, "num_key_value_heads": 2, "intermediate_size": 768,
                          "vocab_size": 1000, "rope_theta": 1e4, "quantization": {"group_size": 32, "bits": 4}})
    assert (c.head_dim, c.n_kv_heads, c.group_size, c.rope_theta, c.rms_eps) == (128, 2, 32, 1e4, 1e-5)


def test_gate_and_up_rows_interleave_in_runs_of_eight_with_zero_padding():
    import torch
    from scratchy_b200.dense import interleave8
    gate, up = torch.arange(20.0).reshape(10, 2), 100 + torch.arange(20.0).reshape(10, 2)
    w = interleave8(gate, up)
    assert w.shape == (32, 2)
    assert torch.equal(w[:8], gate[:8]) and torch.equal(w[8:16], up[:8]) and torch.equal(w[16:18], gate[8:]) and torch.equal(w[24:26], up[8:])
    assert not w[18:24].any() and not w[26:].any()


# ---------------------------------------------------------------------------------------- bookkeeping
def test_sequence_table_hands_out_and_takes_back():
    t = SequenceTable(4, 8, 2)
    a, b = t.open("a"), t.open("b")
    with pytest.raises(OutOfCache):
        t.open("c")
    with pytest.raises(ValueError):
        t.open("a")
    t.extend(a, 8)
    assert len(a.blocks) == 1
    t.advance(a, 8)
    t.extend(a, 1)
    assert len(a.blocks) == 2 and t.free_blocks == 2
    with pytest.raises(OutOfCache):
        t.extend(b, 17)
    assert b.blocks == [] and t.free_blocks == 2          # all or nothing
    t.extend(b, 16)
    assert not set(a.blocks) & set(b.blocks)
    t.close("a")
    assert t.free_blocks == 2 and t.free_slots == 1
    c = t.open("c")
    assert c.slot == a.slot and c.length == 0 and c.blocks == []


def test_blocks_that_the_window_has_passed_go_back():
    from scratchy_b200.sequences import NO_BLOCK
    t = SequenceTable(8, 4, 2, window=6, keep_first=5)                         # the first two blocks stay
    s = t.open("s")
    t.extend(s, 17)
    t.advance(s, 17)                                                           # the next token, 17, sees 12..17 and 0..4
    assert len(s.blocks) == 5 and s.held == 4 and s.blocks[2] == NO_BLOCK and t.free_blocks == 4
    for length in range(18, 60):
        t.extend(s, 1)
        t.advance(s, 1)
        visible = {j // 4 for j in range(length + 1) if length - j < 6 or j < 5}
        held = {i for i, b in enumerate(s.blocks) if b != NO_BLOCK}
        assert visible - {length // 4} <= held <= visible | {length // 4 - 1} and s.held <= t.most_blocks(60, 1)
        assert s.held + t.free_blocks == 8
    t.close("s")
    assert sorted(t._free_blocks) == list(range(8))
    assert SequenceTable(8, 4, 1).most_blocks(60, 1) == 15 and t.most_blocks(9, 100) == 3 and t.most_blocks(1000, 8) == 2 + 4 + 1


def test_generation_beyond_the_cache_with_a_window():
    m = Recorder(num_blocks=9, block_size=4, max_sequences=3)
    m.table = SequenceTable(9, 4, 3, window=6, keep_first=3)
    prompts = [[1, 2, 3] * 10, [4] * 25, [5, 6]]
    assert Engine(m, step_tokens=4).generate(prompts, 20) == [continue_alone(p, 20) for p in prompts]
    assert m.table.free_blocks == 9
    with pytest.raises(ValueError, match="do not fit"):
        Engine(m, step_tokens=100).generate([[1] * 90], 6)                     # in one portion


class Recorder:
    """A model of the serving interface whose greedy token is a function of the sequence so far."""
    vocab = 50

    def __init__(self, num_blocks=64, block_size=4, max_sequences=3, max_portion=1000):
        self.table, self.max_portion = SequenceTable(num_blocks, block_size, max_sequences), max_portion
        self.seen, self.steps = {}, []

    def forward(self, entries, want):
        import torch
        self.steps.append([(seq.name, len(tok)) for seq, tok in entries])
        rows = []
        for (seq, tok), places in zip(entries, want):
            self.table.extend(seq, len(tok))
            past = self.seen.setdefault(seq.name, []) if seq.length else self.seen.update({seq.name: []}) or self.seen[seq.name]
            assert len(past) == seq.length
            for i, t in enumerate(tok):
                past.append(t)
                if i in places:
                    row = torch.zeros(self.vocab)
                    row[self.next_token(past)] = 1.0
                    rows.append(row)
            self.table.advance(seq, len(tok))
        return torch.stack(rows) if rows else None

    @staticmethod
    def next_token(past):
        return (sum(past) * 7 + len(past)) % 50

    def greedy(self, logits):
        return logits.argmax(1).tolist()

    def check_health(self):
        pass


def continue_alone(prompt, n, stop=()):
    past, out = list(prompt), []
    for _ in range(n):
        out.append(Recorder.next_token(past))
        past.append(out[-1])
        if out[-1] in stop:
            break
    return out


@pytest.mark.parametrize("portion,step_tokens", [(1000, 2048), (3, 2048), (1000, 5), (1, 7)])
def test_generation_does_not_depend_on_scheduling(portion, step_tokens):
    prompts = [[1, 2, 3], [4] * 11, [5], [6, 7], list(range(30))]
    m = Recorder(max_portion=portion)
    out = Engine(m, step_tokens=step_tokens).generate(prompts, 6)
    assert out == [continue_alone(p, 6) for p in prompts]
    assert m.table.free_blocks == 64 and m.table.free_slots == 3
    assert all(sum(n for _, n in s) <= max(step_tokens, 3) for s in m.steps)


def test_admission_never_strands_a_running_request():
    m = Recorder(num_blocks=6, block_size=4, max_sequences=3)
    prompts = [[1] * 9, [2] * 9, [3] * 3]
    assert Engine(m).generate(prompts, 6) == [continue_alone(p, 6) for p in prompts]      # 4 + 4 + 3 blocks never fit together
    with pytest.raises(ValueError, match="do not fit"):
        Engine(m).generate([[1] * 20], 6)


def test_stop_tokens_end_a_request_early():
    p = [3, 1, 4]
    full = continue_alone(p, 12)
    stop = full[4]
    assert Engine(Recorder()).generate([p], 12, stop_ids=[stop]) == [continue_alone(p, 12, (stop,))]


def test_requests_are_checked_before_they_run():
    e = Engine(Recorder())
    for prompt, n in (([], 3), ([1], 0), ([50], 3), ([-1], 3)):
        with pytest.raises(ValueError):
            e.submit(prompt, n)


def test_a_step_is_cut_to_the_models_portions_and_keeps_the_order_of_wants():
    whole, cut = Recorder(), Recorder(max_portion=2)
    entries = [("a", [1, 2, 3, 4, 5], [0, 3, 4]), ("b", [6, 7], []), ("c", [8], [0])]
    a, b = Engine(whole).run_step(entries), Engine(cut).run_step(entries)
    assert a.shape == (4, 50) and (a == b).all()
    assert cut.steps == [[("a", 2), ("b", 2), ("c", 1)], [("a", 2)], [("a", 1)]]
    assert Engine(whole).run_step([("a", [9], [])], ["a", "b"]) is None
    assert sorted(whole.table.live) == ["c"]


def test_trace_replay_writes_wanted_rows_and_confirms_every_step(tmp_path, monkeypatch):
    m = Recorder()
    monkeypatch.setattr(registry, "load_model", lambda *a, **k: m)
    monkeypatch.setattr(registry, "prepare_library", lambda directory: None)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": [5, 17, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": [9], "want": []}], "end": []},
             {"step": 7, "entries": [{"id": "x", "tokens": [4], "want": [0]}], "end": ["x"]},
             {"step": 8, "entries": [{"id": "x", "tokens": [4], "want": [0]}], "end": ["x"]}]
    out = io.StringIO()
    args = types.SimpleNamespace(model="m", dtype="bfloat16", out=str(tmp_path), max_tokens=64, max_sequences=2)
    assert trace.run(args, [json.dumps(s) + "\n" for s in steps], out) == 0
    assert out.getvalue().split("\n")[:-1] == [f"done {s['step']}" for s in steps]
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 50).argmax(1).tolist()
    assert read(0) == [Recorder.next_token([5, 17, 3]), Recorder.next_token([5])]
    assert not (tmp_path / "1.f32").exists()
    assert read(7) == [Recorder.next_token([5, 17, 3, 9, 4])]
    assert read(8) == [Recorder.next_token([4])]                     # the name starts afresh after its end


def test_a_number_format_without_a_model_is_refused_with_its_own_code(tmp_path, monkeypatch):
    from scratchy_b200._lib import ScratchyCudaError

    def refuse(*a, **k):
        raise ScratchyCudaError(-4, "no")
    monkeypatch.setattr(registry, "load_model", refuse)
    monkeypatch.setattr(registry, "prepare_library", lambda directory: None)
    args = types.SimpleNamespace(model="m", dtype="float32", out=str(tmp_path), max_tokens=64, max_sequences=2)
    assert trace.run(args, [], io.StringIO()) == 3
