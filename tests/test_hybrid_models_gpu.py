"""The hybrid decoders on the GPU as whole models against their float64 oracles, through their own generation paths: layers,
schedules, batches, padding, greedy generation, recorded graphs, the trace runner.  Every test runs for every design."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import dafovik_oracle, lonulix_oracle
from tests import dafovik_cases, lonulix_cases
from tests.dafovik_cases import rel_rms, worst_row, write_checkpoint

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DESIGNS = {"dafovik": (dafovik_cases, dafovik_oracle), "lonulix": (lonulix_cases, lonulix_oracle)}
ALL = [(d, n) for d in sorted(DESIGNS) for n in sorted(DESIGNS[d][0].CONFIGS)]
each_model = pytest.mark.parametrize("design,name", ALL)
each_design = pytest.mark.parametrize("design", sorted(DESIGNS))

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    memo = {}

    def get(design, name, dtype):
        """(model, configuration, tensors, folder, oracle).  In bf16 the choice of experts is settled by its corrections: a
        rounding may turn a close call, which the oracle does not follow."""
        if (design, name, dtype) not in memo:
            import trimkv_b200 as t
            cases, oracle = DESIGNS[design]
            cfg = cases.CONFIGS[name]
            tensors = cases.random_tensors(cfg, 7, **({"settled": True} if design == "lonulix" and dtype is BF16 else {}))
            path = write_checkpoint(tmp_path_factory.mktemp(name), cfg, tensors)
            memo[(design, name, dtype)] = (t.load_model(path, dtype=dtype, device=DEV), cfg, tensors, path, oracle)
        return memo[(design, name, dtype)]
    return get


def _logit_error(got, want):
    got = got.double().cpu().numpy() if torch.is_tensor(got) else got
    return worst_row(got - got.mean(-1, keepdims=True), want - want.mean(-1, keepdims=True))


MODEL_TOL = {F32: 1e-4, BF16: 0.12}


@pytest.mark.parametrize("dtype", [F32, BF16])
@each_model
def test_model_layers_and_logits(design, name, dtype, models):
    model, cfg, tensors, _, orc = models(design, name, dtype)
    ids = np.random.default_rng(3).integers(0, cfg["vocab"], 60)
    layers, mine = [], []
    want = orc.forward(cfg, tensors, ids, layers)
    cache = model.new_cache()
    cache.open(1)
    got = model.forward_packed(torch.from_numpy(ids).to(DEV), cache, [60], layers_out=mine)
    assert got.dtype is F32 and len(mine) == len(cfg["layers"])
    for a, b in zip(mine, layers):
        assert a.dtype is F32 and rel_rms(a, b) < (5e-6 if dtype is F32 else 3e-2)
    assert _logit_error(got, want) < MODEL_TOL[dtype] and rel_rms(got, want) < MODEL_TOL[dtype] / 3


@pytest.mark.parametrize("dtype", [F32, BF16])
@each_model
def test_model_schedules_agree(design, name, dtype, models):
    """Whole prompts, portions, token by token and mixed batches give the same logits at every position."""
    model, cfg, tensors, _, orc = models(design, name, dtype)
    rng = np.random.default_rng(4)
    lens = [90, 33, 2, 61]
    seqs = [rng.integers(0, cfg["vocab"], n) for n in lens]
    want = [orc.forward(cfg, tensors, s) for s in seqs]
    shared = model.new_cache()                                          # slots are given back and taken again throughout
    for r, s in enumerate(seqs):                                        # alone, then decoding
        for split in (len(s), max(1, len(s) - 40), 1):
            shared.open(1)
            out = [model.forward_packed(torch.from_numpy(s[:split]).to(DEV), shared, [split])]
            out += [model.forward_packed(torch.from_numpy(s[i:i + 1]).to(DEV), shared, [1]) for i in range(split, len(s))]
            assert _logit_error(torch.cat(out), want[r]) < MODEL_TOL[dtype], (r, split)
            shared.close([0])
    for sizes in ([7], [2], [40, 5]):                                   # together, in portions; requests end one by one
        shared.open(4)
        order, at, got = [0, 1, 2, 3], [0] * 4, [[] for _ in lens]
        i = 0
        while order:
            n = [min(sizes[i % len(sizes)] + (r if sizes != [2] else 0), lens[r] - at[r]) for r in order]
            ids = np.concatenate([seqs[r][at[r]:at[r] + m] for r, m in zip(order, n)])
            y = model.forward_packed(torch.from_numpy(ids).to(DEV), shared, n)
            for r, part, m in zip(order, y.split(n), n):
                got[r].append(part)
                at[r] += m
            gone = [p for p, r in enumerate(order) if at[r] == lens[r]]
            if gone:
                shared.close(gone)
                order = [r for p, r in enumerate(order) if p not in gone]
            i += 1
        for r in range(4):
            assert _logit_error(torch.cat(got[r]), want[r]) < MODEL_TOL[dtype], (sizes, r)
    shared.check_status()
    assert len(shared._free) == shared._nslots


@each_design
def test_padding_on_either_side_and_wanted_places(design, models):
    model, cfg, tensors, _, orc = models(design, "mixed", F32)
    rng = np.random.default_rng(5)
    lens = [9, 4, 14]
    seqs = [rng.integers(1, cfg["vocab"], n) for n in lens]
    want = [orc.forward(cfg, tensors, s) for s in seqs]
    for side in ("left", "right"):
        ids, mask = np.zeros((3, 14), np.int64), np.zeros((3, 14), np.int64)
        for r, s in enumerate(seqs):
            sl = slice(14 - len(s), 14) if side == "left" else slice(0, len(s))
            ids[r, sl], mask[r, sl] = s, 1
        ids_d, mask_d = torch.from_numpy(ids).to(DEV), torch.from_numpy(mask).to(DEV)
        full = model(input_ids=ids_d, attention_mask=mask_d).logits
        last = model(input_ids=ids_d, attention_mask=mask_d, logits_to_keep=1).logits
        assert last.shape == (3, 1, cfg["vocab"])
        for r in range(3):
            assert _logit_error(full[r][mask_d[r].bool()], want[r]) < 1e-4
            assert _logit_error(last[r], want[r][-1:]) < 1e-4
    cache = model.new_cache()
    cache.open(2)
    flat = torch.from_numpy(np.concatenate(seqs[:2])).to(DEV)
    some = model.forward_packed(flat, cache, lens[:2], want=[12, 3])
    assert _logit_error(some, np.stack([want[1][3], want[0][3]])) < 1e-4
    assert model.forward_packed(flat, cache, lens[:2], want=[]).shape == (0, cfg["vocab"])


def _greedy_oracle(orc, cfg, tensors, ids, new):
    out = list(ids)
    for _ in range(new):
        out.append(int(orc.forward(cfg, tensors, out)[-1].argmax()))
    return out


@each_design
def test_greedy_generation_through_every_entry_point(design, models):
    model, cfg, tensors, _, orc = models(design, "mixed", F32)
    rng = np.random.default_rng(6)
    lens, new = [12, 5, 23], 24
    seqs = [rng.integers(1, cfg["vocab"], n).tolist() for n in lens]
    want = [_greedy_oracle(orc, cfg, tensors, s, new) for s in seqs]
    ids = torch.zeros(3, 23, dtype=torch.int64)
    mask = torch.zeros(3, 23, dtype=torch.int64)
    for r, s in enumerate(seqs):
        ids[r, 23 - len(s):], mask[r, 23 - len(s):] = torch.tensor(s), 1
    ids, mask = ids.to(DEV), mask.to(DEV)

    def check(out, label):
        for r, s in enumerate(seqs):
            assert out[r, 23 - len(s):].tolist() == want[r], (label, r)
    check(model.generate_greedy(ids, max_new_tokens=new, attention_mask=mask), "greedy")
    check(model.generate_greedy(ids, max_new_tokens=new, attention_mask=mask, prefill_chunk_size=7), "chunked prompt")
    check(model.generate_greedy(ids, max_new_tokens=new, attention_mask=mask, fused_decode=True), "graph-replayed")
    check(model.generate(ids, attention_mask=mask, max_new_tokens=new, do_sample=False, pad_token_id=0), "HF loop")
    model.config.fused_decode_step = True
    try:
        check(model.generate(ids, attention_mask=mask, max_new_tokens=new, do_sample=False, pad_token_id=0), "HF loop, graph-replayed step")
    finally:
        model.config.fused_decode_step = False
    right = torch.zeros_like(ids)
    rmask = torch.zeros_like(mask)
    for r, s in enumerate(seqs):
        right[r, :len(s)], rmask[r, :len(s)] = torch.tensor(s, device=DEV), 1
    out = model.generate_greedy(right, max_new_tokens=new, attention_mask=rmask, prefill_chunk_size=6)
    for r, s in enumerate(seqs):
        assert out[r, 23:].tolist() == want[r][len(s):], ("right padding", r)
    torch.manual_seed(0)                                                # sampling is HF's
    out = model.generate(ids, attention_mask=mask, max_new_tokens=4, do_sample=True, top_k=5, pad_token_id=0)
    assert out.shape == (3, 27) and int(out.max()) < cfg["vocab"]


@each_design
def test_long_decoding_with_a_recorded_graph(design, models):
    """The recorded one-token step over growing windows (arrays move, the graph is recorded again) and wrapped rings, bf16."""
    from trimkv_b200.decoder import GreedyDecoder
    model, cfg, tensors, _, orc = models(design, "mixed", BF16)
    ids = np.random.default_rng(8).integers(0, cfg["vocab"], (2, 150))
    want = [orc.forward(cfg, tensors, s) for s in ids]
    cache = model.new_cache()
    with torch.inference_mode():
        model(input_ids=torch.from_numpy(ids[:, :10]).to(DEV), past_key_values=cache)
        dec = GreedyDecoder(model, cache)
        for i in range(10, 150):
            dec.step(torch.from_numpy(ids[:, i:i + 1]).to(DEV), eager=i < 12)
            assert _logit_error(dec.logits, np.stack([w[i] for w in want])) < MODEL_TOL[BF16], i
    assert dec.graph is not None and cache.row_lengths() == [150, 150]
    dec.close()
    cache.check_status()


@each_design
def test_finished_requests_leave_a_batch(design, models):
    model, cfg, tensors, _, orc = models(design, "odd", F32)
    rng = np.random.default_rng(9)
    seqs = rng.integers(0, cfg["vocab"], (3, 30))
    want = [orc.forward(cfg, tensors, s) for s in seqs]
    cache = model.new_cache()
    model(input_ids=torch.from_numpy(seqs[:, :20]).to(DEV), past_key_values=cache)
    cache.batch_select_indices(torch.tensor([2, 0]))
    for i in range(20, 30):
        got = model(input_ids=torch.from_numpy(seqs[[2, 0], i:i + 1]).to(DEV), past_key_values=cache).logits[:, 0]
        assert _logit_error(got, np.stack([want[2][i], want[0][i]])) < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@each_design
def test_trace_runner_on_a_checkpoint(design, dtype, models, tmp_path):
    _, cfg, tensors, path, orc = models(design, "mixed", getattr(torch, dtype))
    rng = np.random.default_rng(10)
    a, b = rng.integers(0, cfg["vocab"], 40), rng.integers(0, cfg["vocab"], 12)
    steps = [{"step": 0, "entries": [{"id": "b", "tokens": b[:10].tolist(), "want": [9, 2]}, {"id": "a", "tokens": a[:30].tolist(), "want": []}], "end": []}]
    for i in range(10):
        entries = [{"id": "a", "tokens": [int(a[30 + i])], "want": [0]}] + ([{"id": "b", "tokens": [int(b[10 + i])], "want": [0]}] if i < 2 else [])
        steps.append({"step": i + 1, "entries": entries, "end": ["b"] if i == 1 else []})
    steps[-1]["end"] = ["a"]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "52"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(11)]
    wa, wb = orc.forward(cfg, tensors, a), orc.forward(cfg, tensors, b)
    want = {0: wb[[9, 2]], **{i + 1: np.stack([wa[30 + i]] + ([wb[10 + i]] if i < 2 else [])) for i in range(10)}}
    for n, w in want.items():
        got = np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(w.shape).astype(float)
        assert _logit_error(got, w) < MODEL_TOL[getattr(torch, dtype)], n
