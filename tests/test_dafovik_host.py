"""Host side of the hybrid decoder without a GPU: configuration, registry, checkpoints, state-cache bookkeeping, trace
protocol, argument errors of the entry points; and sanity of the float64 oracle its GPU tests compare with."""
import io
import json
import os
import sys
from concurrent.futures import ThreadPoolExecutor

import numpy as np
import pytest
import torch

from oracle import dafovik_oracle as orc
from tests import dafovik_cases as cases


# ------------------------------------------------------------------------------------------------ oracle
def test_recurrence_equals_the_sum_over_the_past():
    rng = np.random.default_rng(0)
    T, H, N, P = 9, 2, 5, 3
    q, k, v = rng.standard_normal((T, H, N)), rng.standard_normal((T, H, N)), rng.standard_normal((T, H, P))
    a = rng.uniform(0.3, 1.0, (T, H))
    o, S = orc.scalar_decay_recurrence(q, k, v, a)
    for t in range(T):
        for h in range(H):
            want = sum(np.prod(a[j + 1:t + 1, h]) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert np.allclose(o[t, h], want)
    o2, S2 = orc.scalar_decay_recurrence(q[4:], k[4:], v[4:], a[4:], orc.scalar_decay_recurrence(q[:4], k[:4], v[:4], a[:4])[1])
    assert np.allclose(o2, o[4:]) and np.allclose(S2, S)


def test_window_counts_the_position_itself():
    T, W = 12, 4
    k = np.zeros((T, 1, 2))
    q = np.ones((T, 1, 2))
    v = np.eye(T)[:, None, :]
    p = orc.window_softmax(q, k, v, 1.0, W)[:, 0]
    for i in range(T):
        seen = np.nonzero(p[i])[0].tolist()
        assert seen == list(range(max(0, i - W + 1), i + 1)) and np.allclose(p[i, seen], 1.0 / len(seen))


def test_rotation_preserves_relative_angles():
    rng = np.random.default_rng(1)
    x, y = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))

    def dot(p, q):
        return float((orc.rotate_half_pairs(x, np.array([p]), 100.0, 6) * orc.rotate_half_pairs(y, np.array([q]), 100.0, 6)).sum())
    assert np.isclose(dot(3, 1), dot(40, 38)) and not np.isclose(dot(3, 1), dot(3, 2))
    assert np.array_equal(orc.rotate_half_pairs(x, np.array([7]), 100.0, 6)[..., 6:], x[..., 6:])


# ------------------------------------------------------------------------------------------------ configuration, checkpoints
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_checkpoint_round_trip_and_registry(name, tmp_path):
    import trimkv_b200 as t
    cfg = cases.CONFIGS[name]
    tensors = cases.random_tensors(cfg, 1)
    path = cases.write_checkpoint(tmp_path / "a", cfg, tensors)
    assert t.model_class(path) is t.DafovikForCausalLM
    model = t.load_model(path, dtype=torch.float32, device="cpu")
    mine = model.checkpoint_tensors()
    assert set(mine) == set(tensors)
    for k, v in mine.items():
        assert np.array_equal(v.detach().numpy(), tensors[k]), k
    for layer in model.model.layers:                                    # padding rows of fused projections stay zero
        assert not layer.mix.proj.weight[layer.mix.proj.used:].any()
    model.save_checkpoint(str(tmp_path / "b"))
    again = t.load_model(str(tmp_path / "b"), dtype=torch.float32, device="cpu")
    assert again.config.checkpoint_dict() == model.config.checkpoint_dict()
    for k, v in again.checkpoint_tensors().items():
        assert torch.equal(v, mine[k]), k


def test_loader_refuses_what_does_not_fit(tmp_path):
    import trimkv_b200 as t
    cfg = cases.CONFIGS["odd"]
    good = cases.random_tensors(cfg)
    for change, word in ((lambda d: d.pop("l1.mix.lk2"), "missing"), (lambda d: d.update(extra=np.zeros(3, np.float32)), "unexpected"),
                         (lambda d: d.update({"l0.norm1": np.zeros(5, np.float32)}), "shape")):
        bad = dict(good)
        change(bad)
        path = cases.write_checkpoint(tmp_path / word, cfg, bad)
        with pytest.raises(ValueError, match=word):
            t.DafovikForCausalLM.from_pretrained(path, dtype=torch.float32)
    with pytest.raises(ValueError, match="float16"):
        t.DafovikForCausalLM.from_pretrained(path, dtype=torch.float16)


def test_config_names_what_it_does_not_know(tmp_path):
    import trimkv_b200 as t
    with pytest.raises(ValueError, match="unknown mixer"):
        t.DafovikConfig(layers=[{"type": "conv", "mixer": {}, "mlp": None}])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        t.DafovikConfig(layers=[{**cases.mamba2(), "mlp": {"kind": "routed", "ff": 8}}])
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(KeyError, match="Other"):
        t.model_class(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "qwen3", "architectures": ["Qwen3ForCausalLM"]}))
    assert t.model_class(str(tmp_path)) is t.TrimKVQwen3ForCausalLM


def test_model_without_a_gpu_raises(tmp_path):
    import trimkv_b200 as t
    from trimkv_b200._lib import TrimKVNativeError
    cfg = cases.CONFIGS["odd"]
    model = t.load_model(cases.write_checkpoint(tmp_path, cfg, cases.random_tensors(cfg)), device="cpu")
    if not torch.cuda.is_available():
        with pytest.raises((TrimKVNativeError, RuntimeError)):
            model(input_ids=torch.zeros(1, 3, dtype=torch.int64))


# ------------------------------------------------------------------------------------------------ state cache
@pytest.fixture
def host_cache(monkeypatch):
    """A HybridStateCache on the CPU whose one native call is restated in torch."""
    from trimkv_b200 import ops, state_cache

    def batch_begin(lens, slots, cu, pos0):
        s = slots.long()
        pos0.copy_(lens[s])
        lens[s] += 1 if cu is None else cu[1:] - cu[:-1]
    monkeypatch.setattr(ops, "batch_begin", batch_begin)
    monkeypatch.setattr(torch.cuda, "is_current_stream_capturing", lambda: False)

    def make(window=10, **kw):
        layers = [state_cache.RecurrentState(2, 3, 4, 3, 5), state_cache.WindowState(1, 64, 64, window), state_cache.RecurrentState(1, 2, 2)]
        return state_cache.HybridStateCache(layers, "cpu", torch.float32, **kw)
    return make


def test_slots_are_reused_and_rows_move_up(host_cache):
    c = host_cache()
    assert c.open(3) == [0, 1, 2]
    c.begin([5, 1, 7])
    slots = list(c._rows)
    c.close([1])
    assert c.row_lengths() == [5, 7] and c._rows == [slots[0], slots[2]]
    assert c.open(1) == [2] and c._rows[2] == slots[1] and c.row_lengths() == [5, 7, 0]
    b = c.begin([2, 1, 4])
    assert b.pos0.tolist() == [5, 7, 0] == b.starts and b.cu.tolist() == [0, 2, 3, 7] and b.max_tokens == 4
    assert c._lens[c._rows].tolist() == c.row_lengths() == [7, 8, 4]
    b = c.begin(None)
    assert b.cu is None and b.pos0.tolist() == [7, 8, 4] and c.get_seq_length() == 9
    assert c.get_cache_length(1) == 9 and c.get_cache_length(0) == 0
    c.batch_select_indices(torch.tensor([2, 0]))
    assert c.row_lengths() == [5, 8] and len(c._free) == c._nslots - 2
    with pytest.raises(ValueError, match="duplicated"):
        c.batch_select_indices([0, 0])


def test_begin_over_some_rows_and_its_errors(host_cache):
    c = host_cache()
    c.open(3)
    c.begin([2, 3, 4])
    b = c.begin([6, 2], rows=[2, 0])
    assert b.slots.tolist() == [c._rows[2], c._rows[0]] and b.starts == [4, 2] and c.row_lengths() == [4, 3, 10]
    for counts, rows in (([0, 1], [0, 1]), ([1, 1], [0, 0]), ([1], [0, 1])):
        with pytest.raises(ValueError):
            c.begin(counts, rows=rows)
    with pytest.raises(ValueError, match="without requests"):
        host_cache().begin([])


def test_growth_keeps_what_is_held(host_cache):
    c = host_cache(window=1000)
    c.open(2)
    assert c.arrays(1)["k"].shape[2] == 64
    c.begin([60, 10])
    for i, d in enumerate(c._data):
        for j, a in enumerate(d.values()):
            a.copy_(torch.arange(a.numel(), dtype=torch.float32).view_as(a) + 1000 * i + j)
    before = [{n: a.clone() for n, a in d.items()} for d in c._data]
    key = c.graph_key()
    assert c.fits(4) and not c.fits(5)
    c.begin([10, 1])                                                    # 70 positions: more rows
    assert c.arrays(1)["k"].shape[2] == 128 and c.graph_key() != key
    assert torch.equal(c.arrays(1)["k"][:, :, :64], before[1]["k"]) and torch.equal(c.arrays(1)["v"][:, :, :64], before[1]["v"])
    c.open(3)                                                           # more slots
    for d, old in zip(c._data, before):
        for n, a in d.items():
            got = a[:2] if n not in ("k", "v") else a[:2, :, :64]
            assert torch.equal(got, old[n]), n
    assert c._lens[c._rows].tolist() == c.row_lengths() == [70, 11, 0, 0, 0]
    small = host_cache(window=10)
    small.open(1)
    small.begin([500])
    assert small.arrays(1)["k"].shape[2] == 10                          # never more rows than the window


def test_window_plan_places_the_history_before_the_new_tokens(host_cache):
    c = host_cache(window=10)
    c.open(3)
    b = c.begin([4, 30, 1])
    start, rows, hist = b.window_plan(10)
    assert start is b.cu and rows == 35 and hist == 0
    b = c.begin([3, 2, 5])
    start, rows, hist = b.window_plan(10)
    assert start.tolist() == [0, 7, 18] and rows == 24 and hist == 9    # histories 4, 9 (of 30), 1
    assert b.window_plan(1)[1:] == (10, 0) and b.window_plan(10)[0] is start


def test_decode_batches_are_static_until_the_batch_changes(host_cache):
    c = host_cache()
    c.open(2)
    c.begin([3, 4])
    b1 = c.begin(None)
    key = c.graph_key()
    b2 = c.begin(None)
    assert b2.slots is b1.slots and b2.pos0 is b1.pos0 and c.graph_key() == key
    snap = c.snapshot_counters()
    c.advance(1)
    c.restore_counters(snap)
    assert c.row_lengths() == [5, 6]
    c.close([0])
    assert c.begin(None).slots.tolist() == [c._rows[0]] and c.graph_key() != key


# ------------------------------------------------------------------------------------------------ trace protocol
class _EchoModel:
    """Stands for a model: the logits of a token are [token id, position, request's first token]."""
    device = "cpu"

    class _Cache:
        def __init__(self):
            self.past, self.closed = [], []

        def open(self, n):
            self.past += [[] for _ in range(n)]

        def close(self, rows):
            self.closed.append(sorted(rows))
            self.past = [p for i, p in enumerate(self.past) if i not in set(rows)]

        def check_status(self):
            pass

    def new_cache(self, capacity_tokens=0):
        return self._Cache()

    def forward_packed(self, ids, cache, lengths, rows, want):
        out, at = [], 0
        for i, n in enumerate(lengths):
            past = cache.past[i if rows is None else rows[i]]
            for t in ids[at:at + n].tolist():
                past.append(t)
                out.append([t, len(past) - 1, past[0]])
            at += n
        return torch.tensor(out, dtype=torch.float32)[want]


def test_trace_runner_protocol(tmp_path, monkeypatch, capsys):
    from trimkv_b200 import build, registry, trace
    model = _EchoModel()
    monkeypatch.setattr(build, "build", lambda *a, **k: None)
    monkeypatch.setattr(registry, "load_model", lambda *a, **k: model)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}, {"id": "b", "tokens": [9], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [8], "want": []}, {"id": "a", "tokens": [4], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [7], "want": [0]}], "end": []},
             {"step": 3, "entries": [], "end": ["b"]},
             {"step": 4, "entries": [{"id": "a", "tokens": [1, 2], "want": [1, 0]}], "end": ["a"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace.main(["--model", "x", "--out", str(tmp_path), "--max-tokens", "9"]) == 0
    assert capsys.readouterr().out.split("\n")[:-1] == [f"done {i}" for i in range(5)]
    read = {int(f.split(".")[0]): np.fromfile(tmp_path / f, "<f4").reshape(-1, 3).tolist() for f in os.listdir(tmp_path)}
    assert read == {0: [[5, 0, 5], [3, 2, 5]], 2: [[7, 2, 9]], 4: [[2, 1, 1], [1, 0, 1]]}


def test_trace_needs_requests_of_unequal_length():
    from trimkv_b200.trace import TraceSession
    with pytest.raises(TypeError, match="unequal"):
        TraceSession(torch.nn.Linear(1, 1))


# ------------------------------------------------------------------------------------------------ entry points
def _argument_errors():
    from trimkv_b200 import _lib, build
    build.build()
    lib = _lib.lib()
    one = 16                                                            # a non-NULL, aligned address that is never used
    assert lib.tkv_embed_stream(None, one, 4, one, None, 1, 8, 1.0, 0, None, None) == -1
    assert lib.tkv_postnorm_add(one, one, one, None, 1, 8, 1e-6, 1.0, 1.0, 1, None) == -2           # f16
    assert lib.tkv_gated_norm(one, 4, one, 8, None, 0, one, 1, 1, 8, 1e-6, 0, 0, None) == -1           # stride below a row
    assert lib.tkv_rotate_qk(one, 64, one, None, one, 1, 1, 2, 8, 7, one, 1.0, 0, None) == -1       # odd rotary dims
    assert lib.tkv_conv_silu(one, 4, one, one, one, one, one, one, one, 1, 1, 8, 4, 0, None) == -1
    assert lib.tkv_linrec_scan(one, 8, one, 8, one, 8, None, None, None, None, one, one, one, None, one, 1, 1, 1, 8, 8, 0, None) == -1
    assert lib.tkv_linrec_chunk_workspace_bytes(1, 64, 64, 2, 12, 8, 0) == -1 and lib.tkv_linrec_chunk_workspace_bytes(1, 64, 64, 2, 16, 8, 2) == -1
    assert lib.tkv_linrec_chunk_workspace_bytes(4, 64, 256, 64, 64, 64, 0) == 0 and lib.tkv_linrec_chunk_workspace_bytes(1, 4096, 4096, 2, 64, 64, 0) > 0
    assert lib.tkv_diff_decode_workspace_bytes(2, 4, 2, 300, 192, 64, 0) == 0
    assert lib.tkv_diff_decode(one, one, one, 9, one, one, one, 0.1, 1.0, 1e-6, one, 4, one, None, 0, 1, 4, 3, 8, 8, 64, 64, 0, None) == -1
    assert lib.tkv_diff_decode(one, one, one, 9, one, one, one, 0.1, 1.0, 1e-6, one, 4, one, None, 0, 1, 4, 2, 8, 8, 64, 64, 0, None) == -1
    assert b"workspace" in lib.tkv_last_error()
    assert lib.tkv_batch_begin(one, None, None, one, 1, None) == -1


def test_argument_errors_are_reported_without_a_gpu():
    # in a thread of its own: the library's last error is kept per thread, and another test looks at the main thread's
    with ThreadPoolExecutor(1) as pool:
        pool.submit(_argument_errors).result()
