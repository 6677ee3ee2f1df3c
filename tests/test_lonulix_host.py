"""Host side of the latent-attention / HGRN2 decoder without a GPU: configuration, registry, checkpoints, state cache, argument
errors; and sanity of the float64 oracle its GPU tests compare with."""
import json
from concurrent.futures import ThreadPoolExecutor

import numpy as np
import pytest
import torch

from oracle import lonulix_oracle as orc
from tests import lonulix_cases as cases
from tests.dafovik_cases import write_checkpoint


# ------------------------------------------------------------------------------------------------ oracle
def test_recurrence_equals_the_sum_over_the_past():
    rng = np.random.default_rng(0)
    T, H, N, P = 9, 2, 5, 3
    q, v = rng.standard_normal((T, H, N)), rng.standard_normal((T, H, P))
    f = rng.uniform(0.01, 1.0, (T, H, N))
    o, S = orc.channel_decay_recurrence(q, f, v)
    for t in range(T):
        for h in range(H):
            want = sum(((q[t, h] * np.prod(f[j + 1:t + 1, h], axis=0)) @ (1 - f[j, h])) * v[j, h] for j in range(t + 1))
            assert np.allclose(o[t, h], want)
    o2, S2 = orc.channel_decay_recurrence(q[4:], f[4:], v[4:], orc.channel_decay_recurrence(q[:4], f[:4], v[:4])[1])
    assert np.allclose(o2, o[4:]) and np.allclose(S2, S)


def test_window_counts_the_position_itself():
    m = orc.window_mask(9, 4)
    for i in range(9):
        assert np.nonzero(m[i])[0].tolist() == list(range(max(0, i - 3), i + 1))


def test_rotation_turns_neighbours_by_relative_angles():
    rng = np.random.default_rng(1)
    x, y = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))

    def dot(p, q):
        return float((orc.rotate_neighbours(x, np.array([float(p)]), 50.0, 6) * orc.rotate_neighbours(y, np.array([float(q)]), 50.0, 6)).sum())
    assert np.isclose(dot(3, 1), dot(40, 38)) and not np.isclose(dot(3, 1), dot(3, 2))
    z = orc.rotate_neighbours(x, np.array([2.0]), 50.0, 6)
    assert np.array_equal(z[:, 6:], x[:, 6:])
    assert np.allclose(z[0, :2], [x[0, 0] * np.cos(2) - x[0, 1] * np.sin(2), x[0, 1] * np.cos(2) + x[0, 0] * np.sin(2)])


def test_routing_rules():
    z = np.log(np.array([0.1, 0.2, 0.05, 0.3, 0.25, 0.1]))
    chosen, w = orc.route(z, np.zeros(6), 2, 3, 3, 1.0)
    assert chosen.tolist() == [3, 4] and np.allclose(w, np.array([0.3, 0.25]) / 0.55)
    # groups of two: the best scores are 0.2, 0.3, 0.25; with one group kept its weaker member is chosen too
    assert sorted(orc.route(z, np.zeros(6), 2, 3, 1, 1.0)[0].tolist()) == [2, 3]
    # the correction decides the choice (all choice scores negative), the weights do not see it
    chosen, w = orc.route(z, np.array([-1.0, -1.9, -3, -3, -3, -3]), 2, 3, 1, 2.0)
    assert chosen.tolist() == [0, 1] and np.allclose(w, 2.0 * np.array([0.1, 0.2]) / 0.3)


def test_group_norm_parts_are_independent():
    x = np.random.default_rng(2).standard_normal((1, 12))
    y = x.copy()
    y[:, 4:8] *= 100.0
    a, b = orc.group_rms(x, np.ones(12), 3, 0.0), orc.group_rms(y, np.ones(12), 3, 0.0)
    assert np.allclose(a, b) and not np.allclose(orc.group_rms(x, np.ones(12), 1, 0.0), orc.group_rms(y, np.ones(12), 1, 0.0))


# ------------------------------------------------------------------------------------------------ configuration, checkpoints
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_checkpoint_round_trip_and_registry(name, tmp_path):
    import trimkv_b200 as t
    cfg = cases.CONFIGS[name]
    tensors = cases.random_tensors(cfg, 1)
    path = write_checkpoint(tmp_path / "a", cfg, tensors)
    assert t.model_class(path) is t.LonulixForCausalLM
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
    for change, word in ((lambda d: d.pop("l0.mlp.e4.up"), "missing"), (lambda d: d.update({"l1.mlp.router": np.zeros((3, 37), np.float32)}), "unexpected"),
                         (lambda d: d.update({"l0.rg1": np.zeros((37, 36), np.float32)}), "shape")):
        bad = dict(good)
        change(bad)
        path = write_checkpoint(tmp_path / word, cfg, bad)
        with pytest.raises(ValueError, match=word):
            t.LonulixForCausalLM.from_pretrained(path, dtype=torch.float32)


def test_config_names_what_it_does_not_know():
    import trimkv_b200 as t
    with pytest.raises(ValueError, match="unknown mixer"):
        t.LonulixConfig(layers=[{"type": "retention", "mixer": {}, "mlp": None}])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        t.LonulixConfig(layers=[{**cases.hgrn2(), "mlp": {"kind": "other"}}])
    with pytest.raises(ValueError, match="norm groups"):
        t.LonulixConfig(width=10, norm={"eps": 1e-6, "groups": 3})
    for bad in (dict(groups=(4, 2)), dict(top=7), dict(groups=(3, 4))):
        with pytest.raises(ValueError, match="experts"):
            t.LonulixForCausalLM(t.LonulixConfig(**{k: v for k, v in cases.config([(cases.hgrn2(), cases.experts(**bad))]).items() if k != "architecture"}))


def test_new_models_initialise_their_own_parts():
    import trimkv_b200 as t
    cfg = {k: v for k, v in cases.CONFIGS["mixed"].items() if k != "architecture"}
    m = t.LonulixForCausalLM(t.LonulixConfig(**cfg))
    for k, v in m.checkpoint_tensors().items():
        assert torch.isfinite(v).all(), k
        if k.endswith(("norm1", "norm2", "dq.norm", "dkv.norm", "mix.norm", "final.norm")):
            assert torch.equal(v, torch.ones_like(v)), k
        elif not k.endswith((".b", "correction", "lower")):
            assert v.std() > 0, k
    assert m.model.norm.centre == 1.0 and json.loads(json.dumps(m.config.checkpoint_dict()))["postln_alpha"] == 2.2


# ------------------------------------------------------------------------------------------------ state cache
def test_latent_rows_grow_and_keep_their_places(monkeypatch):
    from trimkv_b200 import ops, state_cache

    def batch_begin(lens, slots, cu, pos0):
        s = slots.long()
        pos0.copy_(lens[s])
        lens[s] += 1 if cu is None else cu[1:] - cu[:-1]
    monkeypatch.setattr(ops, "batch_begin", batch_begin)
    monkeypatch.setattr(torch.cuda, "is_current_stream_capturing", lambda: False)
    c = state_cache.HybridStateCache([state_cache.LatentState(128, 1000), state_cache.RecurrentState(2, 3, 4), state_cache.LatentState(64, 5)],
                                     "cpu", torch.float32)
    c.open(2)
    c.begin([60, 10])
    a = c.arrays(0)["latent"]
    assert a.shape == (2, 64, 128) and c.arrays(2)["latent"].shape == (2, 5, 64)
    a.copy_(torch.arange(a.numel(), dtype=torch.float32).view_as(a))
    old, key = a.clone(), c.graph_key()
    c.begin([10, 1])                                                    # 70 positions: more rows
    assert c.arrays(0)["latent"].shape == (2, 128, 128) and c.graph_key() != key
    assert torch.equal(c.arrays(0)["latent"][:, :64], old) and c.arrays(2)["latent"].shape == (2, 5, 64)
    c.open(2)                                                           # more slots
    assert torch.equal(c.arrays(0)["latent"][:2, :64], old)
    assert [c.get_cache_length(i) for i in range(3)] == [70, 0, 5]


# ------------------------------------------------------------------------------------------------ entry points
def _argument_errors():
    from trimkv_b200 import _lib, build
    build.build()
    lib = _lib.lib()
    one = 16                                                            # a non-NULL, aligned address that is never used
    assert lib.tkv_gated_sum_norm(one, one, None, None, 0, None, 0, None, one, None, 1, 10, 3, 1e-6, 1.0, 0, None) == -1     # 10 in 3 parts
    assert lib.tkv_gated_sum_norm(one, one, one, None, 2, None, 0, None, one, None, 1, 9, 3, 1e-6, 1.0, 0, None) == -1       # weights missing
    assert lib.tkv_swiglu(one, 15, one, 1, 8, 0, None) == -1
    assert lib.tkv_chanrec_scan(one, one, one, 8, one, one, one, one, one, None, one, 1, 2, 8, 8, 0, None) == -1             # rows too short
    assert lib.tkv_chanrec_step(one, one, one, 16, one, one, None, 1e-6, one, one, one, one, 1, 2, 8, 8, 0, None) == -1
    assert lib.tkv_chanrec_chunk_workspace_bytes(1, 64, 2, 12, 8, 0) == -1 and lib.tkv_chanrec_chunk_workspace_bytes(1, 64, 2, 16, 8, 2) == -1
    assert lib.tkv_chanrec_chunk_workspace_bytes(8, 4096, 64, 64, 64, 0) == 0 and lib.tkv_chanrec_chunk_workspace_bytes(1, 4096, 2, 64, 64, 0) > 0
    assert lib.tkv_rotate_pairs(one, 64, None, one, 1, 1, 2, 8, 4, 6, one, 0, None) == -1                                    # part beyond the head
    assert lib.tkv_latent_prep(one, 64, one, one, 1e-6, 8, 8, 4, 3, one, one, one, 5, None, None, None, one, one, 1, 1, 0, 5, 0, None) == -1
    assert lib.tkv_latent_decode_workspace_bytes(2, 4, 520, 64, 300, 0) == -1 and lib.tkv_latent_decode_workspace_bytes(2, 4, 64, 32, 300, 2) == -1
    assert lib.tkv_latent_decode_workspace_bytes(2, 4, 64, 32, 300, 0) > 0
    assert lib.tkv_latent_decode(one, 8, 8, one, 8, 8, one, one, 9, one, one, 1.0, one, 8, 8, None, 0, 1, 4, 8, 8, 8, 0, None) == -1
    assert b"workspace" in lib.tkv_last_error()
    assert lib.tkv_moe_route(one, 8, one, 4, 8, 0, 3, 4, 1, 1.0, one, one, one, one, None, one, None) == -1                  # three of two open experts
    assert lib.tkv_moe_route(one, 8, one, 200, 8, 0, 2, 4, 1, 1.0, one, one, one, one, None, one, None) == -1                # counts missing
    assert lib.tkv_moe_gemm(one, 7, 4, one, one, one, one, 4, 2, 8, 8, 0, 0, None, None) == -1


def test_argument_errors_are_reported_without_a_gpu():
    with ThreadPoolExecutor(1) as pool:                                 # the library's last error is kept per thread
        pool.submit(_argument_errors).result()
