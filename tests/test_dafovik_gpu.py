"""Mechanisms of the Dafovik decoder on the GPU, each alone, against the float64 oracle (whole models:
``test_hybrid_models_gpu``).  fp32 runs compare to rounding of fp32, bf16 runs to rounding of their 16-bit operands; where random data
would hide a fault (a far key among many, a window's edge), one key is made to stand out."""
import numpy as np
import pytest
import torch

from oracle import dafovik_oracle as orc
from tests import dafovik_cases as cases
from tests.dafovik_cases import rel_rms, worst_row

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32
# Worst row of a mixer.  bf16: its projections and products round to 8 bits, softmax scores of a few units amplify that (the
# mean error is asserted at a third of it).
TOL = {F32: 2e-5, BF16: 2.5e-2}


def on_gpu(x, dtype=F32):
    return torch.as_tensor(np.ascontiguousarray(x)).to(dtype).to(DEV)


def as_held(x, dtype):
    """What the device holds of x, in float64."""
    return torch.as_tensor(np.asarray(x)).to(dtype).double().numpy()


def cache_of(*layers, dtype, **kw):
    from trimkv_b200.state_cache import HybridStateCache
    return HybridStateCache(list(layers), DEV, dtype, **kw)


def splits(T, sizes):
    out, at, i = [], 0, 0
    while at < T:
        n = min(sizes[i % len(sizes)], T - at)
        out.append((at, at + n))
        at, i = at + n, i + 1
    return out


# ------------------------------------------------------------------------------------------------ elementwise steps
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [37, 72, 512, 5000])
def test_embedding_residual_and_norms(dtype, width):
    from trimkv_b200 import ops
    rng = np.random.default_rng(width)
    table, y, w = as_held(rng.standard_normal((50, width)), dtype), as_held(rng.standard_normal((7, width)) * 3, dtype), rng.standard_normal(width) * 0.3
    w = as_held(w, F32)
    ids = torch.tensor([3, 49, 0, 7, 7, 12, 31], device=DEV)
    status = ops.new_status(DEV)
    stream, copy = torch.empty(7, width, device=DEV), torch.empty(7, width, dtype=dtype, device=DEV)
    ops.embed_stream(ids, on_gpu(table, dtype), stream, copy, status)
    assert torch.equal(stream.double().cpu(), torch.from_numpy(table[ids.cpu().numpy()])) and torch.equal(copy.float(), stream)
    want = orc.post_norm_residual(table[ids.cpu().numpy()], y, w, 0.6, 1e-5)
    ops.postnorm_add(stream, on_gpu(y, dtype), on_gpu(w), copy, 1e-5, 0.6, 1.0)
    assert worst_row(stream, want) < 1e-6 and torch.equal(copy, stream.to(dtype))       # the stream is fp32 for every type
    out = torch.empty(3, width, dtype=dtype, device=DEV)
    rows = torch.tensor([6, 0, 2], dtype=torch.int32, device=DEV)
    ops.stream_norm(stream, rows, on_gpu(w), out, 1e-5, 1.0)
    assert worst_row(out, orc.centred_norm(want[[6, 0, 2]], w, 1e-5)) < (1e-6 if dtype is F32 else 4e-3)
    assert ops.read_status(status) == 0
    ops.embed_stream(torch.tensor([50], device=DEV), on_gpu(table, dtype), stream[:1], None, status)
    assert ops.read_status(status) == 3 and not stream[:1].any()
    u = on_gpu(y, dtype)
    ops.gelu_tanh(u)
    assert worst_row(u, orc.gelu_tanh(y)) < (1e-6 if dtype is F32 else 4e-3)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("groups,length", [(1, 40), (3, 7), (4, 64), (2, 1032)])
def test_gated_group_norms(dtype, groups, length):
    from trimkv_b200 import ops
    rng = np.random.default_rng(length)
    C, T = groups * length, 5
    y = as_held(rng.standard_normal((T, C)) * np.repeat(10.0 ** np.arange(groups), length), dtype)     # groups of unlike size
    zw = as_held(rng.standard_normal((T, C + 24)), dtype)
    z, w = zw[:, 8:8 + C], as_held(rng.standard_normal(C), F32)
    out, zd = torch.empty(T, C, dtype=dtype, device=DEV), on_gpu(zw, dtype)[:, 8:8 + C]
    ops.gated_norm(on_gpu(y, dtype), zd, on_gpu(w), out, groups, 1e-4, gate_first=True)
    assert worst_row(out, orc.grouped_gated_norm(y, z, w, groups, 1e-4)) < (2e-6 if dtype is F32 else 5e-3)
    ops.gated_norm(on_gpu(y, dtype), zd, None, out, groups, 1e-4, gate_first=False)
    want = orc.unit_rms(y.reshape(T, groups, length), 1e-4).reshape(T, C) * orc.silu(z)
    assert worst_row(out, want) < (2e-6 if dtype is F32 else 5e-3)


# ------------------------------------------------------------------------------------------------ rotation, convolution
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,rot", [(2, 16, 16), (3, 10, 6), (2, 64, 32), (1, 8, 2)])
def test_rotation_far_from_the_start(dtype, heads, dim, rot):
    from trimkv_b200 import ops
    from trimkv_b200.mixers import RetentionMixer
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(dim)
    mix = RetentionMixer(8, heads, dim, 4, [0.5] * heads, rot, 1e6, 1e-6)
    c = cache_of(RecurrentState(heads, dim, 4), dtype=dtype)
    c.open(2)
    c.begin([70001, 1])
    b = c.begin([5, 9])
    raw = as_held(rng.standard_normal((14, 2 * heads * dim + 8)), dtype)
    out = torch.empty(14, 2 * heads * dim, dtype=dtype, device=DEV)
    ops.rotate_qk(on_gpu(raw, dtype), out, b, heads, dim, rot, mix._freq(torch.device(DEV)), dim ** -0.5)
    pos = np.concatenate([70001 + np.arange(5), 1 + np.arange(9)]).astype(float)
    hd = heads * dim
    q = orc.rotate_half_pairs(raw[:, :hd].reshape(14, heads, dim), pos, 1e6, rot).reshape(14, hd)
    k = orc.rotate_half_pairs(raw[:, hd:2 * hd].reshape(14, heads, dim), pos, 1e6, rot).reshape(14, hd) * dim ** -0.5
    tol = 1e-6 if dtype is F32 else 4e-3                                # the angle keeps its accuracy at large positions
    assert worst_row(out[:, :hd], q) < tol and worst_row(out[:, hd:], k) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("taps,channels", [(1, 16), (2, 13), (4, 40), (4, 9), (7, 24)])
def test_convolution_over_portions(dtype, taps, channels):
    from trimkv_b200 import ops
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(taps * channels)
    lens = [45, 3, 20]
    x = [as_held(rng.standard_normal((n, channels)), dtype) for n in lens]
    w, bias = as_held(rng.standard_normal((channels, taps)), F32), as_held(rng.standard_normal(channels), F32)
    c = cache_of(RecurrentState(1, 1, 1, taps, channels), dtype=dtype)
    c.open(5)
    c.close([0, 2])                                                     # slots out of order
    c.arrays(0)["conv"].fill_(float("nan"))                             # whatever an earlier request left
    got, at = [[] for _ in lens], [0] * 3
    for step in ([2, 1, 7], [17, 1, 2], [2, 1, 1], [24, 0, 10]):
        rows = [i for i, n in enumerate(step) if n]
        b = c.begin([step[i] for i in rows], rows)
        part = np.concatenate([x[i][at[i]:at[i] + step[i]] for i in rows])
        wide = on_gpu(np.concatenate([part, part[:, :8]], 1), dtype)
        out = torch.empty(len(part), channels, dtype=dtype, device=DEV)
        if b.cu is None:
            continue
        ops.conv_silu(wide[:, :channels], c.arrays(0)["conv"], on_gpu(w), on_gpu(bias), out, b)
        o = 0
        for i in rows:
            got[i].append(out[o:o + step[i]])
            o, at[i] = o + step[i], at[i] + step[i]
    for i in range(3):
        assert worst_row(torch.cat(got[i]), orc.causal_conv_silu(x[i], w, bias)) < (2e-6 if dtype is F32 else 5e-3)


# ------------------------------------------------------------------------------------------------ recurrence
def _recurrence_case(rng, lens, heads, groups, n, p, dtype, far=None):
    T = sum(lens)
    q, k, v = (as_held(rng.standard_normal(s), dtype) for s in ((T, groups, n), (T, groups, n), (T, heads, p)))
    logd = -np.exp(rng.uniform(-7, 0.5, (T, heads)))
    if far is not None:                                                 # one early key that only one late query asks for
        src, dst = far
        k[:, :, 0] = 0
        q[:, :, 0] = 0
        k[src, :, 0] = q[dst, :, 0] = 32.0
        logd[:, 0] = -1e-5
    return q, k, v, as_held(logd, F32), as_held(rng.uniform(0.1, 1.5, (T, heads)), F32), as_held(rng.standard_normal(heads), F32)


def _oracle_recurrence(q, k, v, logd, scale, skip, lens):
    heads, groups = v.shape[1], q.shape[1]
    grp = np.arange(heads) // (heads // groups)
    out, states, at = [], [], 0
    for n in lens:
        s = slice(at, at + n)
        o, S = orc.scalar_decay_recurrence(q[s][:, grp], k[s][:, grp], scale[s][:, :, None] * v[s], np.exp(logd[s]))
        out.append(o + skip[:, None] * v[s])
        states.append(S)
        at += n
    return np.concatenate(out), states


@pytest.mark.parametrize("dtype,scan", [(F32, True), (BF16, True), (BF16, False)])
@pytest.mark.parametrize("heads,groups,n,p", [(2, 1, 64, 64), (4, 2, 56, 24), (2, 2, 128, 128), (1, 1, 8, 136), (2, 1, 200, 72), (6, 3, 16, 8), (2, 1, 72, 72), (4, 2, 128, 64)])
def test_recurrence_ragged_and_in_portions(dtype, scan, heads, groups, n, p):
    from trimkv_b200 import ops
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(n * p)
    lens = [300, 64, 2, 1]
    q, k, v, logd, scale, skip = _recurrence_case(rng, lens, heads, groups, n, p, dtype, far=(3, 298))
    want, states = _oracle_recurrence(q, k, v, logd, scale, skip, lens)
    start = np.cumsum([0] + lens)
    for sizes in ([1000], [2, 63, 65], [64], [129, 140]):
        c = cache_of(RecurrentState(heads, n, p), dtype=dtype)
        c.open(len(lens))
        c.arrays(0)["state"].fill_(float("nan"))
        got = np.full(want.shape, np.nan)
        parts = [splits(L, sizes) for L in lens]
        for i in range(max(len(x) for x in parts)):
            rows = [r for r in range(len(lens)) if i < len(parts[r])]
            sel = np.concatenate([np.arange(start[r] + parts[r][i][0], start[r] + parts[r][i][1]) for r in rows])
            b = c.begin([parts[r][i][1] - parts[r][i][0] for r in rows], rows)
            out = torch.empty(len(sel), heads * p, dtype=dtype, device=DEV)
            ops.linrec(on_gpu(q[sel].reshape(len(sel), -1), dtype), on_gpu(k[sel].reshape(len(sel), -1), dtype), on_gpu(v[sel].reshape(len(sel), -1), dtype),
                       c.arrays(0)["state"], b, out, groups, log_decay=on_gpu(logd[sel]), v_scale=on_gpu(scale[sel]), skip=on_gpu(skip),
                       force_scan=scan)
            got[sel] = out.double().cpu().numpy().reshape(len(sel), heads, p)
        tol = 2e-5 if dtype is F32 else 6e-3
        assert worst_row(got, want) < tol, sizes
        for r, S in enumerate(states):                                  # the state is fp32 whatever the operands' type
            assert rel_rms(c.arrays(0)["state"][c._rows[r]], S) < 3e-5, (sizes, r)


@pytest.mark.parametrize("n,p", [(32, 40), (128, 64), (96, 136), (200, 64)])
def test_recurrence_cut_into_segments(n, p):
    """Few heads and a long sequence: segments run side by side and start from the chained states."""
    from trimkv_b200 import _lib, ops
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(5)
    lens, heads = [1500, 70, 777], 2
    assert _lib.lib().tkv_linrec_chunk_workspace_bytes(3, 1500, sum(lens), heads, n, p, 0) > 0
    q, k, v, logd, scale, skip = _recurrence_case(rng, lens, heads, 1, n, p, BF16, far=(1, 1499))
    want, states = _oracle_recurrence(q, k, v, logd, scale, skip, lens)
    c = cache_of(RecurrentState(heads, n, p), dtype=BF16)
    c.open(3)
    c.arrays(0)["state"].fill_(float("nan"))
    start, got = np.cumsum([0] + lens), np.full(want.shape, np.nan)
    for lo, hi in ((0, 0.4), (0.4, 1.0)):                               # the second call starts from a state
        cut = [(int(L * lo), int(L * hi)) for L in lens]
        sel = np.concatenate([np.arange(start[r] + a, start[r] + z) for r, (a, z) in enumerate(cut)])
        b = c.begin([z - a for a, z in cut])
        out = torch.empty(len(sel), heads * p, dtype=BF16, device=DEV)
        ops.linrec(on_gpu(q[sel].reshape(len(sel), -1), BF16), on_gpu(k[sel].reshape(len(sel), -1), BF16), on_gpu(v[sel].reshape(len(sel), -1), BF16),
                   c.arrays(0)["state"], b, out, 1, log_decay=on_gpu(logd[sel]), v_scale=on_gpu(scale[sel]), skip=on_gpu(skip))
        got[sel] = out.double().cpu().numpy().reshape(len(sel), heads, p)
    assert worst_row(got, want) < 6e-3
    for r, S in enumerate(states):
        assert rel_rms(c.arrays(0)["state"][c._rows[r]], S) < 3e-5


def test_recurrence_with_constant_decay_per_head():
    from trimkv_b200 import ops
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(6)
    T, heads, n, p = 200, 3, 16, 24
    decay = np.array([0.5, 1 - 2.0 ** -9, 1.0])
    q, k, v = (as_held(rng.standard_normal((T, heads, s)), BF16) for s in (n, n, p))
    want, _ = orc.scalar_decay_recurrence(q, k, v, np.tile(decay, (T, 1)))
    args = [on_gpu(a.reshape(T, -1), BF16) for a in (q, k, v)]
    for scan in (False, True):
        c = cache_of(RecurrentState(heads, n, p), dtype=BF16)
        c.open(1)
        out = torch.empty(T, heads * p, dtype=BF16, device=DEV)
        ops.linrec(*args, c.arrays(0)["state"], c.begin([T]), out, heads, head_decay=on_gpu(decay), head_log_decay=on_gpu(np.log(decay)), force_scan=scan)
        assert worst_row(out.view(T, heads, p), want) < 6e-3


# ------------------------------------------------------------------------------------------------ mixers: prompts and decoding
def _mixer(layer, width, seed, dtype, eps=3e-6):
    """(module on the GPU, oracle of the same mixer)."""
    from trimkv_b200.modeling_dafovik import MIXERS
    cfg = cases.config([layer], width=width)
    t = {k[len("l0.mix."):]: v for k, v in cases.random_tensors(cfg, seed).items() if k.startswith("l0.mix.")}
    mix = MIXERS[layer["type"]](width, layer["mixer"], eps)
    with torch.no_grad():
        for name, p in mix.checkpoint().items():
            p.copy_(torch.from_numpy(t[name]))
    mix = mix.to(dtype).to(DEV)
    t64 = {k: v.astype(np.float64) for k, v in t.items()}
    return mix, lambda h: orc.MIXERS[layer["type"]](h, t64, layer["mixer"], eps)


MIXER_CASES = {
    "retention": cases.retention(heads=2, dim=16, vdim=24, rot=8),
    "retention_odd": cases.retention(heads=3, dim=10, vdim=7, rot=4),
    "retention_wide": cases.retention(heads=1, dim=96, vdim=272, rot=96),
    "mamba2": cases.mamba2(heads=4, vdim=16, state=24, groups=2, conv=3, norm_groups=2),
    "mamba2_odd": cases.mamba2(heads=3, vdim=5, state=9, groups=3, conv=5, norm_groups=1),
    "mamba2_norm_across_heads": cases.mamba2(heads=4, vdim=8, state=16, groups=1, conv=4, norm_groups=2),
    "mamba2_one_tap": cases.mamba2(heads=2, vdim=64, state=128, groups=2, conv=1, norm_groups=4),
    "attention": cases.attention(heads=4, kv_heads=2, dim=24, vdim=40, window=19),
    "attention_odd": cases.attention(heads=3, kv_heads=3, dim=13, vdim=9, window=6),
    "attention_wide": cases.attention(heads=2, kv_heads=1, dim=136, vdim=200, window=21),
    "attention_full_tiles": cases.attention(heads=2, kv_heads=1, dim=64, vdim=128, window=64),
    "attention_large_heads": cases.attention(heads=2, kv_heads=2, dim=128, vdim=128, window=50),
    "attention_many_queries": cases.attention(heads=18, kv_heads=2, dim=32, vdim=64, window=33),
    "attention_small_values": cases.attention(heads=2, kv_heads=2, dim=100, vdim=16, window=44),
    "attention_negative_scale": cases.attention(heads=2, kv_heads=1, dim=16, vdim=16, window=44, scale=-0.3),
    "attention_window_of_one": cases.attention(heads=2, kv_heads=1, dim=16, vdim=16, window=1),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(MIXER_CASES))
def test_mixer_prompts_portions_and_decoding(name, dtype):
    """Unequal requests in one batch, cut in several ways, slots dirty from earlier use, then token by token."""
    mix, oracle = _mixer(MIXER_CASES[name], 40, 3, dtype)
    rng = np.random.default_rng(11)
    lens = [150, 37, 5]
    x = [as_held(rng.standard_normal((n, 40)), dtype) for n in lens]
    want = [oracle(h) for h in x]
    tol = TOL[dtype] * (2.4 if name.startswith("attention") and dtype is BF16 else 1)
    for sizes, decode_from in (([1000], 1000), ([1000], 4), ([2], 30), ([64, 3, 17], 120), ([50], 100)):
        c = cache_of(mix.state(), dtype=dtype)
        c.open(4)
        c.close([1])
        for a in c.arrays(0).values():
            a.fill_(float("nan"))
        got, at = [np.full(w.shape, np.nan) for w in want], [0, 0, 0]
        i = 0
        while any(a < n for a, n in zip(at, lens)):
            rows = [r for r in range(3) if at[r] < lens[r]]
            step = {}
            for r in rows:
                step[r] = 1 if at[r] >= decode_from else min(sizes[i % len(sizes)], lens[r] - at[r], max(decode_from - at[r], 1))
            ids = np.concatenate([x[r][at[r]:at[r] + step[r]] for r in rows])
            b = c.begin([step[r] for r in rows], rows)
            with torch.inference_mode():
                y = mix(on_gpu(ids, dtype), b, c.arrays(0)).double().cpu().numpy()
            o = 0
            for r in rows:
                got[r][at[r]:at[r] + step[r]] = y[o:o + step[r]]
                o, at[r] = o + step[r], at[r] + step[r]
            i += 1
        c.check_status()
        for r in range(3):
            assert worst_row(got[r], want[r]) < tol and rel_rms(got[r], want[r]) < tol / 3, (sizes, decode_from, r)


def _edge_case(window, T, heads, kv_heads, dim, vdim, targets):
    """Projection rows in which, for every (query i, key j) of ``targets``, key j of map 1 stands out for query i (a code of
    its own in the key's dims), and every value is distinct."""
    rng = np.random.default_rng(window + T)
    q, k = rng.standard_normal((T, heads, 2, dim)) * 0.05, rng.standard_normal((T, kv_heads, 2, dim)) * 0.05
    v = rng.standard_normal((T, kv_heads, vdim))
    for c, (i, j) in enumerate(targets):
        q[i, :, 0, c % dim] += 4.0
        k[j, :, 0, c % dim] += 4.0
    return np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window,T", [(1, 20), (2, 40), (43, 260), (127, 400), (128, 400), (129, 520), (300, 700)])
def test_keys_just_inside_and_just_outside_the_window(window, T, dtype):
    from trimkv_b200 import ops
    from trimkv_b200.state_cache import WindowState
    heads, kv_heads, dim, vdim, scale, diff = 4, 2, 32, 48, 1.0, 0.2
    ends = sorted({window - 1, window, 127, 128, 129, 255, 256, 257, T - 1, T - 2} & set(range(1, T)))
    targets = []
    for i in ends:                                                      # last key inside, first key outside, the first token
        targets += [(i, j) for j in (i - window + 1, i - window, 0, i) if 0 <= j <= i]
    raw = as_held(_edge_case(window, T, heads, kv_heads, dim, vdim, targets), dtype)
    pad = np.concatenate([raw, np.zeros((T, 8))], 1)
    gate = as_held(np.random.default_rng(1).standard_normal((T, heads)), dtype)
    qn, kn, eps, lam = np.full(dim, 2.0), np.full(dim, 1.5), 1e-6, 0.45
    nq, nk = heads * 2 * dim, kv_heads * 2 * dim
    q = orc.unit_rms(raw[:, :nq].reshape(T, heads, 2, dim), eps) * qn
    k = orc.unit_rms(raw[:, nq:nq + nk].reshape(T, kv_heads, 2, dim), eps) * kn
    if dtype is BF16:
        q, k = as_held(q, BF16), as_held(k, BF16)
    v = raw[:, nq + nk:].reshape(T, kv_heads, vdim)
    a1, a2 = (orc.window_softmax(q[:, :, m], k[:, :, m], v, scale, window) for m in (0, 1))
    want = orc.differential_combine(a1, a2, lam, diff, eps) * orc.sigmoid(gate)[:, :, None]
    lam_d = torch.full((1,), lam, device=DEV)

    def run(pieces):
        c = cache_of(WindowState(kv_heads, 64, 64, window), dtype=dtype)
        c.open(1)
        outs = []
        for lo, hi in pieces:
            b = c.begin([hi - lo])
            out = torch.empty(hi - lo, heads * vdim, dtype=dtype, device=DEV)
            ops.diff_attention(on_gpu(pad[lo:hi], dtype), on_gpu(gate[lo:hi], dtype), on_gpu(qn), on_gpu(kn), c.arrays(0)["k"],
                               c.arrays(0)["v"], b, lam_d, diff, scale, eps, out, heads, dim, vdim, window)
            outs.append(out)
        c.check_status()
        return torch.cat(outs).view(T, heads, vdim)
    tol = 2e-5 if dtype is F32 else 2.5e-2
    cut = max(1, T - max(30, min(window + 5, 140)))
    for pieces in ([(0, T)], splits(T, [97, 2, 33]), [(0, cut)] + [(i, i + 1) for i in range(cut, T)]):
        got = run(pieces)
        assert worst_row(got, want) < tol, pieces[:3]
    # the edge matters: with a window one shorter or longer the planted keys change the result by far more
    if window > 1:
        for other in (window - 1, window + 1):
            b1 = orc.window_softmax(q[:, :, 0], k[:, :, 0], v, scale, other)
            b2 = orc.window_softmax(q[:, :, 1], k[:, :, 1], v, scale, other)
            assert worst_row(orc.differential_combine(b1, b2, lam, diff, eps) * orc.sigmoid(gate)[:, :, None], want) > 0.2


def test_decode_over_many_chunks_of_a_ring():
    """A window of several split-KV chunks, sequences below, at and beyond it, prompt longer than the ring."""
    layer = cases.attention(heads=6, kv_heads=2, dim=40, vdim=72, window=700, scale=0.2)
    mix, oracle = _mixer(layer, 48, 4, BF16)
    rng = np.random.default_rng(2)
    lens, tail = [1400, 702, 300, 260], 6
    x = [as_held(rng.standard_normal((n + tail, 48)), BF16) for n in lens]
    c = cache_of(mix.state(), dtype=BF16)
    c.open(4)
    with torch.inference_mode():
        mix(on_gpu(np.concatenate([a[:n] for a, n in zip(x, lens)]), BF16), c.begin(lens), c.arrays(0))
        got = [mix(on_gpu(np.stack([a[n + s] for a, n in zip(x, lens)]), BF16), c.begin(None), c.arrays(0)).double().cpu().numpy() for s in range(tail)]
    c.check_status()
    for r, (a, n) in enumerate(zip(x, lens)):
        assert worst_row(np.stack([g[r] for g in got]), oracle(a)[n:]) < 2.5e-2, r
