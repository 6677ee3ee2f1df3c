"""Mechanisms of the latent-attention / HGRN2 decoder on the GPU, each alone, against the float64 oracle (whole models:
``test_hybrid_models_gpu``).  fp32 runs compare to rounding of fp32, bf16 runs to rounding of their 16-bit operands; where random
data would hide a fault (a far key among many, a window's edge), one key is made to stand out."""
import numpy as np
import pytest
import torch

from oracle import lonulix_oracle as orc
from tests import lonulix_cases as cases
from tests.dafovik_cases import rel_rms, worst_row
from tests.test_dafovik_gpu import as_held, cache_of, on_gpu, splits

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32
TOL = {F32: 2e-5, BF16: 2.5e-2}                                         # worst row of a mixer, as for the other hybrid mixers


# ------------------------------------------------------------------------------------------------ stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,groups", [(36, 3), (72, 1), (192, 6), (512, 4), (4608, 2), (9000, 9), (2500, 5)])
def test_gated_sum_norm_and_final_norm(width, groups, dtype):
    from trimkv_b200 import ops
    rng = np.random.default_rng(width)
    T = 7
    sizes = np.repeat(10.0 ** np.arange(groups), width // groups) ** 0.3                   # parts of unlike size
    table = as_held(rng.standard_normal((50, width)) * sizes, dtype)
    ids = np.array([3, 49, 0, 7, 7, 12, 31])
    stream, copy = torch.empty(T, width, device=DEV), torch.empty(T, width, dtype=dtype, device=DEV)
    ops.embed_stream(torch.from_numpy(ids).to(DEV), on_gpu(table, dtype), stream, copy, None, 1.7)
    x = table[ids] * 1.7
    assert worst_row(stream, x) < 1e-6 and torch.equal(copy, stream.to(dtype))
    w, bias = as_held(1 + 0.3 * rng.standard_normal(width), F32), as_held(rng.standard_normal(width), F32)
    y, zw = as_held(rng.standard_normal((T, width)) * 3, dtype), as_held(rng.standard_normal((T, width + 24)), dtype)
    gate = on_gpu(zw, dtype)[:, 8:8 + width]
    want = orc.group_rms(2.5 * x + orc.sigmoid(zw[:, 8:8 + width] + bias) * y, w, groups, 1e-4)
    ops.gated_sum_norm(stream, on_gpu(y, dtype), on_gpu(w), copy, groups, 1e-4, 2.5, gate, on_gpu(bias))
    assert worst_row(stream, want) < 1e-6 and torch.equal(copy, stream.to(dtype))       # the stream is fp32 for every type
    ungated = orc.group_rms(0.5 * want + y, w, groups, 1e-4)
    ops.gated_sum_norm(stream, on_gpu(y, dtype), on_gpu(w), None, groups, 1e-4, 0.5)
    assert worst_row(stream, ungated) < 1e-6
    out = torch.empty(3, width, dtype=dtype, device=DEV)
    ops.stream_norm(stream, torch.tensor([6, 0, 2], dtype=torch.int32, device=DEV), on_gpu(w), out, 1e-4, 0.0, groups)
    assert worst_row(out, orc.group_rms(ungated[[6, 0, 2]], w, groups, 1e-4)) < (1e-6 if dtype is F32 else 4e-3)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [36, 200])
def test_expert_rows_are_added_up_in_the_residual(width, dtype):
    from trimkv_b200 import ops
    rng = np.random.default_rng(width)
    T, R, top = 5, 9, 3
    x, rows = as_held(rng.standard_normal((T, width)), F32), as_held(rng.standard_normal((R, width)), dtype)
    place = np.array([[0, -1, 4], [8, 7, 6], [-1, -1, -1], [2, 2, 5], [1, 3, -1]])
    cw = as_held(rng.uniform(0.1, 2, (T, top)), F32)
    y = sum(cw[:, c:c + 1] * np.where(place[:, c:c + 1] < 0, x, rows[place[:, c]]) for c in range(top))
    w = as_held(rng.standard_normal(width), F32)
    stream, copy = on_gpu(x), torch.empty(T, width, dtype=dtype, device=DEV)
    ops.gated_sum_norm(stream, on_gpu(rows, dtype), on_gpu(w), copy, 2, 1e-6, 1.3, place=torch.tensor(place, dtype=torch.int32, device=DEV), choice_weight=on_gpu(cw))
    assert worst_row(stream, orc.group_rms(1.3 * x + y, w, 2, 1e-6)) < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_gated_unit_and_head_norm(dtype):
    from trimkv_b200 import ops
    rng = np.random.default_rng(0)
    for ff, extra in ((40, 24), (13, 1)):
        u = as_held(rng.standard_normal((6, 2 * ff + extra)) * 2, dtype)
        out = torch.empty(6, ff, dtype=dtype, device=DEV)
        ops.swiglu(on_gpu(u, dtype), out)
        assert worst_row(out, orc.silu(u[:, :ff]) * u[:, ff:2 * ff]) < (1e-6 if dtype is F32 else 5e-3)
    for heads, p in ((4, 24), (3, 7), (2, 136), (1, 300)):
        y, w = as_held(rng.standard_normal((6, heads * p)), dtype), as_held(rng.standard_normal(p), F32)
        out = torch.empty(6, heads * p, dtype=dtype, device=DEV)
        ops.gated_norm(on_gpu(y, dtype), None, on_gpu(w), out, heads, 1e-3)
        assert worst_row(out, orc.rms(y.reshape(6, heads, p), w, 1e-3).reshape(6, -1)) < (2e-6 if dtype is F32 else 5e-3)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,head_len,offset,dims", [(2, 24, 8, 16), (3, 10, 3, 6), (2, 192, 128, 64), (1, 8, 0, 2)])
def test_rotation_of_neighbours_far_from_the_start(heads, head_len, offset, dims, dtype):
    from trimkv_b200 import ops
    from trimkv_b200.mixers import rotary_frequencies
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(head_len)
    c = cache_of(RecurrentState(1, 8, 8), dtype=dtype)
    c.open(2)
    c.begin([70001, 1])
    b = c.begin([5, 9])
    raw = as_held(rng.standard_normal((14, heads * head_len)), dtype)
    x = on_gpu(raw, dtype)
    ops.rotate_pairs(x, b, heads, head_len, offset, dims, rotary_frequencies(1e6, dims).to(DEV))
    pos = np.concatenate([70001 + np.arange(5), 1 + np.arange(9)]).astype(float)
    want = raw.reshape(14, heads, head_len).copy()
    want[..., offset:offset + dims] = orc.rotate_neighbours(want[..., offset:offset + dims], pos, 1e6, dims)
    assert worst_row(x, want.reshape(14, -1)) < (1e-6 if dtype is F32 else 4e-3)          # the angle keeps its accuracy


# ------------------------------------------------------------------------------------------------ channel-decay recurrence
def _gates_case(rng, T, heads, n, p, dtype, kind):
    """Projections of q, f, v side by side, bias, lower bound.  ``far``: one early value that one late query asks for, in a
    channel that forgets nothing in between.  ``shut``: gates near zero in some channels and places (decays far below what a
    product over a block can hold), beside channels that keep everything.  ``low``: gates around a tenth for a while, which a
    product over 32 tokens cannot hold and one over 16 can."""
    zq, zf, v = (as_held(rng.standard_normal(s), dtype) for s in ((T, heads, n), (T, heads, n), (T, heads, p)))
    bias, lower = rng.standard_normal((heads, n)) + 1.5, np.clip(rng.uniform(-0.3, 0.9, (heads, n)), 0.0, 1.0)
    if kind == "far":
        bias[:, 0] = 0.0
        lower[:, 0] = 0.0
        zq[:, :, 0] = -30.0                                             # silu of it is nothing
        zf[:, :, 0] = 20.0                                              # keeps, writes nothing
        zf[3, :, 0] = -20.0                                             # written once
        zq[T - 2, :, 0] = 64.0
    if kind == "shut":
        lower[:, ::2] = 0.0
        zf[T // 4:T // 2, :, ::4] = -30.0
        zf[:, :, 1] = 40.0
        zf[T // 3, :, 1] = -6.0
        zf[5:9, :, 2 % n] = -90.0
    if kind == "low":
        lower[:, 1::2] = 0.0
        zf[T // 5:T // 2, :, 1::2] = -2.5 - bias[:, 1::2]
    return zq, as_held(zf, dtype), v, as_held(bias, F32), as_held(lower, F32)


def _recurrence_oracle(zq, zf, v, bias, lower, lens):
    out, states, at = [], [], 0
    for n in lens:
        s = slice(at, at + n)
        o, S = orc.channel_decay_recurrence(orc.silu(zq[s]), orc.forget_gate(zf[s], bias, lower), v[s])
        out.append(o)
        states.append(S)
        at += n
    return np.concatenate(out), states


def _run_recurrence(c, b, sel, zq, zf, v, bias, lower, dtype, scan=False):
    from trimkv_b200 import ops
    n, heads, dim, p = len(sel), zq.shape[1], zq.shape[2], v.shape[2]
    u = on_gpu(np.concatenate([a[sel].reshape(n, -1) for a in (zq, zf, v)], 1), dtype)
    out = torch.empty(n, heads * p, dtype=dtype, device=DEV)
    ops.chanrec(u[:, :heads * dim], u[:, heads * dim:2 * heads * dim], u[:, 2 * heads * dim:], on_gpu(bias.reshape(-1)), on_gpu(lower.reshape(-1)),
                c.arrays(0)["state"], b, out, force_scan=scan)
    return out.double().cpu().numpy().reshape(n, heads, p)


@pytest.mark.parametrize("kind", ["far", "shut", "low"])
@pytest.mark.parametrize("dtype,scan", [(F32, True), (BF16, True), (BF16, False)])
@pytest.mark.parametrize("heads,n,p", [(2, 64, 64), (4, 56, 24), (1, 128, 128), (1, 8, 136), (2, 200, 72), (6, 16, 8), (2, 72, 80)])
def test_recurrence_ragged_and_in_portions(heads, n, p, dtype, scan, kind):
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(n * p)
    lens = [300, 64, 2, 1]
    args = _gates_case(rng, sum(lens), heads, n, p, dtype, kind)
    if kind == "far":                                                   # the late query is the first request's
        args[0][298, :, 0], args[0][sum(lens) - 2, :, 0] = 64.0, -30.0
    want, states = _recurrence_oracle(*args, lens)
    if kind == "far":
        assert np.abs(want[298]).mean() > 5 * np.median(np.abs(want))
    start = np.cumsum([0] + lens)
    for sizes in ([1000], [2, 63, 65], [33, 16, 31]):
        c = cache_of(RecurrentState(heads, n, p), dtype=dtype)
        c.open(len(lens))
        c.arrays(0)["state"].fill_(float("nan"))                        # whatever an earlier request left
        got = np.full(want.shape, np.nan)
        parts = [splits(L, sizes) for L in lens]
        for i in range(max(len(x) for x in parts)):
            rows = [r for r in range(len(lens)) if i < len(parts[r])]
            sel = np.concatenate([np.arange(start[r] + parts[r][i][0], start[r] + parts[r][i][1]) for r in rows])
            b = c.begin([parts[r][i][1] - parts[r][i][0] for r in rows], rows)
            got[sel] = _run_recurrence(c, b, sel, *args, dtype, scan)
        assert worst_row(got, want) < (2e-5 if dtype is F32 else 6e-3), sizes
        for r, S in enumerate(states):                                  # the state is fp32 whatever the operands' type
            assert rel_rms(c.arrays(0)["state"][c._rows[r]], S) < 3e-5, (sizes, r)


@pytest.mark.parametrize("kind", ["far", "shut", "low"])
@pytest.mark.parametrize("n,p", [(32, 40), (128, 64), (96, 136), (200, 64)])
def test_recurrence_cut_into_segments(n, p, kind):
    """Few heads and a long sequence: segments run side by side and start from the chained states."""
    from trimkv_b200 import _lib
    from trimkv_b200.state_cache import RecurrentState
    rng = np.random.default_rng(5)
    lens, heads = [1500, 70, 777], 2
    assert _lib.lib().tkv_chanrec_chunk_workspace_bytes(3, 600, heads, n, p, 0) > 0
    args = _gates_case(rng, sum(lens), heads, n, p, BF16, kind)
    if kind == "far":
        args[0][1499, :, 0], args[0][sum(lens) - 2, :, 0] = 64.0, -30.0
    want, states = _recurrence_oracle(*args, lens)
    c = cache_of(RecurrentState(heads, n, p), dtype=BF16)
    c.open(3)
    c.arrays(0)["state"].fill_(float("nan"))
    start, got = np.cumsum([0] + lens), np.full(want.shape, np.nan)
    for lo, hi in ((0, 0.4), (0.4, 1.0)):                               # the second call starts from a state
        cut = [(int(L * lo), int(L * hi)) for L in lens]
        sel = np.concatenate([np.arange(start[r] + a, start[r] + z) for r, (a, z) in enumerate(cut)])
        got[sel] = _run_recurrence(c, c.begin([z - a for a, z in cut]), sel, *args, BF16)
    assert worst_row(got, want) < 6e-3
    for r, S in enumerate(states):
        assert rel_rms(c.arrays(0)["state"][c._rows[r]], S) < 3e-5


# ------------------------------------------------------------------------------------------------ latent attention
def _edge_case(window, T, heads, dim, rot, vdim, rank, targets, dtype):
    """Queries and down-projection rows in which, for every (query i, key j) of ``targets``, key j stands out for query i by a
    code of its own in the latent, which W_uk maps to the key."""
    rng = np.random.default_rng(window + T)
    q, c, r = rng.standard_normal((T, heads, dim + rot)) * 0.2, rng.standard_normal((T, rank)) * 0.05, rng.standard_normal((T, rot)) * 0.2
    uk, uv = rng.standard_normal((heads, dim, rank)) * 0.05, rng.standard_normal((heads, vdim, rank)) / np.sqrt(rank)
    codes = min(dim, rank)
    for h in range(heads):
        uk[h, np.arange(codes), np.arange(codes)] += 1.0
    for k, (i, j) in enumerate(targets):
        q[i, :, k % codes] += 3.0
        c[j, k % codes] += 3.0
    return [as_held(a, dtype) for a in (q, c, r, uk, uv)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window,T", [(3, 32, 16, 40, 48, 1, 20), (3, 32, 16, 40, 48, 2, 40), (2, 40, 8, 24, 72, 43, 260), (2, 32, 64, 128, 128, 127, 400),
                                                              (2, 128, 64, 128, 64, 128, 400), (1, 72, 32, 64, 136, 129, 520), (18, 24, 16, 16, 40, 300, 700)])
def test_keys_just_inside_and_just_outside_the_window(heads, dim, rot, vdim, rank, window, T, dtype):
    from trimkv_b200 import ops
    from trimkv_b200.mixers import rotary_frequencies
    from trimkv_b200.state_cache import LatentState
    scale, eps, base = 0.5, 1e-6, 500.0
    ends = sorted({window - 1, window, 127, 128, 129, 255, 256, 257, T - 1, T - 2} & set(range(1, T)))
    targets = []
    for i in ends:                                                      # last key inside, first key outside, the first token
        targets += [(i, j) for j in (i - window + 1, i - window, 0, i) if 0 <= j <= i]
    q, c_raw, r_raw, uk, uv = _edge_case(window, T, heads, dim, rot, vdim, rank, targets, dtype)
    pos = np.arange(T, dtype=float)
    c = as_held(orc.rms(c_raw, 1.0, eps), dtype)
    kr, qr = orc.rotate_neighbours(r_raw, pos, base, rot), orc.rotate_neighbours(q[..., dim:], pos, base, rot)
    k, v = np.einsum("hdc,tc->thd", uk, c), np.einsum("hpc,tc->thp", uv, c)
    want = orc.two_part_attention(q[..., :dim], qr, k, kr, v, scale, window)
    freq, qn, kn = rotary_frequencies(base, rot).to(DEV), torch.ones(8, device=DEV), torch.ones(rank, device=DEV)
    u = np.concatenate([np.ones((T, 8)), c_raw, r_raw, np.zeros((T, -(rank + rot) % 8))], 1)
    ukv = on_gpu(np.concatenate([uk.reshape(-1, rank), uv.reshape(-1, rank)]), dtype)

    def run(pieces):
        cache = cache_of(LatentState(-(-rank // 64) * 64 + -(-rot // 64) * 64, window), dtype=dtype)
        cache.open(2)
        cache.close([0])
        cache.arrays(0)["latent"].fill_(float("nan"))                   # whatever an earlier request left
        outs = []
        for lo, hi in pieces:
            b = cache.begin([hi - lo])
            n, ring = hi - lo, cache.arrays(0)["latent"]
            _, lin = ops.latent_prep(on_gpu(u[lo:hi], dtype), qn, kn, eps, rot, rot, freq, ring, b, window)
            qd = on_gpu(q[lo:hi].reshape(n, -1), dtype)
            out = torch.empty(n, heads * vdim, dtype=dtype, device=DEV)
            if b.cu is None:
                q3 = qd.view(n, heads, dim + rot)
                q_abs = torch.bmm(q3[:, :, :dim].transpose(0, 1), ukv[:heads * dim].view(heads, dim, rank))
                o = torch.empty_like(q_abs)
                ops.latent_decode(q_abs.transpose(0, 1), q3, rot, freq, ring, b, scale, o.transpose(0, 1), rot)
                out = torch.bmm(o, ukv[heads * dim:].view(heads, vdim, rank).transpose(1, 2)).transpose(0, 1).reshape(n, -1)
            else:
                ops.rotate_pairs(qd, b, heads, dim + rot, dim, rot, freq)
                ops.latent_prefill(qd, torch.mm(lin[:, :rank], ukv.t()), lin, b, scale, out, heads, dim, rot, vdim, rank, window)
            outs.append(out)
        cache.check_status()
        return torch.cat(outs).view(T, heads, vdim)
    tol = 2e-5 if dtype is F32 else 3e-2
    cut = max(1, T - max(30, min(window + 5, 140)))
    for pieces in ([(0, T)], splits(T, [97, 2, 33]), [(0, cut)] + [(i, i + 1) for i in range(cut, T)]):
        assert worst_row(run(pieces), want) < tol, pieces[:3]
    # the edge matters: with a window one shorter or longer the planted keys change the result by far more
    if window > 1:
        for other in (window - 1, window + 1):
            assert worst_row(orc.two_part_attention(q[..., :dim], qr, k, kr, v, scale, other), want) > 0.2


def test_prompt_rows_beyond_a_request_do_not_poison_it():
    """The last key tile of a request reaches into the next request's rows: NaN there must stay there."""
    from trimkv_b200 import ops
    from trimkv_b200.state_cache import LatentState
    rng = np.random.default_rng(3)
    heads, dim, rot, vdim, rank, lens = 2, 16, 16, 24, 16, [40, 50]
    T = sum(lens)
    q, kv = as_held(rng.standard_normal((T, heads * (dim + rot))), BF16), as_held(rng.standard_normal((T, heads * (dim + vdim))), BF16)
    lin = as_held(rng.standard_normal((T, 128)), BF16)
    kv[lens[0]:], lin[lens[0]:] = np.nan, np.nan
    c = cache_of(LatentState(128, 30), dtype=BF16)
    c.open(2)
    b = c.begin(lens)
    out = torch.empty(T, heads * vdim, dtype=BF16, device=DEV)
    ops.latent_prefill(on_gpu(q, BF16), on_gpu(kv, BF16), on_gpu(lin, BF16), b, 0.3, out, heads, dim, rot, vdim, rank, 30)
    n = lens[0]
    q3, k3 = q[:n].reshape(n, heads, dim + rot), kv[:n]
    want = orc.two_part_attention(q3[..., :dim], q3[..., dim:], k3[:, :heads * dim].reshape(n, heads, dim), lin[:n, 64:64 + rot],
                                  k3[:, heads * dim:].reshape(n, heads, vdim), 0.3, 30)
    assert worst_row(out[:n], want.reshape(n, -1)) < 2e-2


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("tokens", [1, 5, 128, 129, 700])
@pytest.mark.parametrize("real,same,top,groups,keep", [(7, 2, 3, 3, 2), (16, 0, 4, 1, 1), (1, 0, 1, 1, 1), (6, 6, 12, 4, 4), (40, 24, 8, 8, 3), (300, 20, 33, 10, 5)])
def test_routing(real, same, top, groups, keep, tokens):
    from trimkv_b200 import ops
    rng = np.random.default_rng(real * tokens)
    E = real + same
    z = as_held(rng.standard_normal((tokens, E)) * 2, F32)
    corr = as_held(rng.standard_normal(E) * 0.2 - 1.5, F32)             # choice scores below zero
    place, weight, src, off = (a.cpu().numpy() for a in ops.moe_route(on_gpu(z), on_gpu(corr), same, top, groups, keep, 2.5))
    owner = np.searchsorted(off, np.arange(off[-1]), side="right") - 1
    assert off[0] == 0 and (np.diff(off) >= 0).all() and off.shape == (real + 1,)
    seen = []
    for t in range(tokens):
        chosen, w = orc.route(z[t], corr, top, groups, keep, 2.5)
        rows = place[t]
        mine = {int(e): float(x) for e, x in zip(chosen, w)}
        real_rows = rows[rows >= 0]
        assert sorted(owner[real_rows].tolist()) == sorted(e for e in mine if e < real), t
        assert (src[real_rows] == t).all()
        for r, x in zip(rows, weight[t]):
            if r >= 0:
                assert abs(x - mine[int(owner[r])]) < 2e-6 * 2.5
        assert np.allclose(sorted(weight[t][rows < 0]), sorted(x for e, x in mine.items() if e >= real), atol=5e-6)
        seen += real_rows.tolist()
    assert sorted(seen) == list(range(int(off[-1])))                    # every row belongs to one choice


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,k", [(40, 72), (8, 8), (264, 136), (13, 9), (128, 64), (600, 200)])
@pytest.mark.parametrize("counts", [[3, 0, 1, 0], [1], [0, 0, 130, 257, 5, 128], [40] * 7])
def test_grouped_products(counts, n, k, dtype):
    from trimkv_b200 import ops
    rng = np.random.default_rng(n * k + len(counts))
    R, E, T = sum(counts), len(counts), 19
    off = torch.tensor(np.concatenate([[0], np.cumsum(counts)]), dtype=torch.int32, device=DEV)
    w = as_held(rng.standard_normal((E, n, k)) / np.sqrt(k), dtype)
    x, src = as_held(rng.standard_normal((T, k)), dtype), rng.integers(0, T, R)
    e = np.repeat(np.arange(E), counts)
    up = np.einsum("rk,rnk->rn", x[src], w[e])
    spare = 11                                                          # rows nobody owns stay as they are
    out = torch.full((R + spare, n), 7.0, dtype=dtype, device=DEV)
    ops.moe_gemm(on_gpu(x, dtype), on_gpu(w, dtype), off, out, src=torch.tensor(np.concatenate([src, np.zeros(spare)]), dtype=torch.int32, device=DEV), act="gelu")
    tol = 3e-6 if dtype is F32 else 5e-3
    assert worst_row(out[:R], orc.gelu_erf(up)) < tol and bool((out[R:] == 7.0).all())
    rows = as_held(rng.standard_normal((R + spare, k)), dtype)
    status = ops.new_status(DEV)
    ops.moe_gemm(on_gpu(rows, dtype), on_gpu(w, dtype), off, out, status=status)
    assert worst_row(out[:R], np.einsum("rk,rnk->rn", rows[:R], w[e])) < tol and ops.read_status(status) == 0


def test_grouped_product_of_many_tiles():
    """More tiles than CTAs, two accumulators and the ring of stages used again and again; wide column tiles."""
    from trimkv_b200 import ops
    gen = torch.Generator(device=DEV).manual_seed(0)
    counts = [700, 0, 1, 129, 3000, 128, 64, 2000]
    R, E, n, k = sum(counts), len(counts), 5000, 328
    off = torch.tensor(np.concatenate([[0], np.cumsum(counts)]), dtype=torch.int32, device=DEV)
    w = torch.randn(E, n, k, generator=gen, device=DEV).to(BF16)
    a, src = torch.randn(500, k, generator=gen, device=DEV).to(BF16), torch.randint(0, 500, (R,), generator=gen, device=DEV).int()
    out, status = torch.empty(R, n, dtype=BF16, device=DEV), ops.new_status(DEV)
    ops.moe_gemm(a, w, off, out, src=src, status=status)
    for e in range(E):
        lo, hi = int(off[e]), int(off[e + 1])
        if hi > lo:
            want = a[src[lo:hi].long()].float() @ w[e].float().t()
            assert float((out[lo:hi].float() - want).abs().max()) < 0.6 and rel_rms(out[lo:hi], want.double().cpu().numpy()) < 3e-3, e
    assert ops.read_status(status) == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [dict(), dict(count=5, top=2, ff=13, identity=1, groups=None), dict(count=8, top=8, ff=24, identity=4, groups=(2, 2)),
                                   dict(count=30, top=5, ff=136, identity=2, groups=(8, 3), scale=0.5)])
def test_expert_layer(shape, dtype):
    """The choice is made from the layer's input as the device holds it, so a rounding turns no choice."""
    from trimkv_b200 import ops
    from trimkv_b200.modeling_lonulix import FEED_FORWARDS
    width, spec = 40, cases.experts(**shape)
    t = {k[len("l0.mlp."):]: v for k, v in cases.random_tensors(cases.config([(cases.hgrn2(), spec)], width=width, groups=1), 5).items() if k.startswith("l0.mlp.")}
    mod = FEED_FORWARDS["moe"](width, spec)
    with torch.no_grad():
        for name, p in mod.checkpoint().items():
            p.copy_(torch.from_numpy(t[name]))
    mod = mod.to(dtype).to(DEV)
    t64 = {k: v.astype(np.float64) for k, v in t.items()}
    for T in (1, 3, 150):
        x = as_held(np.random.default_rng(T).standard_normal((T, width)), dtype)
        with torch.inference_mode():
            y, _ = mod(on_gpu(x, dtype))
        stream = on_gpu(x)
        ops.gated_sum_norm(stream, y.rows, torch.ones(width, device=DEV), None, 1, 0.0, 0.0, place=y.place, choice_weight=y.weight)
        want = orc.rms(orc.expert_mlp(x, t64, spec), 1.0, 0.0)
        assert worst_row(stream, want) < (2e-5 if dtype is F32 else 1.5e-2), T


# ------------------------------------------------------------------------------------------------ mixers: prompts and decoding
def _mixer(layer, width, seed, dtype, eps=3e-6):
    """(module on the GPU, oracle of the same mixer)."""
    from trimkv_b200.modeling_lonulix import MIXERS
    cfg = cases.config([(layer, None)], width=width, groups=1)
    t = {k[len("l0.mix."):]: v for k, v in cases.random_tensors(cfg, seed).items() if k.startswith("l0.mix.")}
    mix = MIXERS[layer["type"]](width, layer["mixer"], eps)
    with torch.no_grad():
        for name, p in mix.checkpoint().items():
            p.copy_(torch.from_numpy(t[name]))
    mix = mix.to(dtype).to(DEV)
    t64 = {k: v.astype(np.float64) for k, v in t.items()}
    return mix, lambda h: orc.MIXERS[layer["type"]](h, t64, layer["mixer"], eps)


MIXER_CASES = {
    "latent": cases.latent(),
    "latent_odd": cases.latent(heads=3, dim=9, rot_dim=6, vdim=7, q_rank=13, kv_rank=11, window=6),
    "latent_window_of_one": cases.latent(window=1),
    "latent_full_tiles": cases.latent(heads=2, dim=128, rot_dim=64, vdim=128, q_rank=64, kv_rank=128, window=64, scale=0.07),
    "latent_wide_values": cases.latent(heads=2, dim=40, rot_dim=32, vdim=104, kv_rank=72, window=50),
    "latent_wide_keys": cases.latent(heads=2, dim=104, rot_dim=8, vdim=32, kv_rank=200, window=44),
    "latent_many_heads": cases.latent(heads=37, dim=16, rot_dim=16, vdim=16, q_rank=40, kv_rank=320, window=33),
    "latent_large_rank": cases.latent(heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=512, window=90),
    "latent_beyond_the_fast_forms": cases.latent(heads=2, dim=136, rot_dim=136, vdim=136, kv_rank=600, window=21, scale=0.05),
    "latent_negative_scale": cases.latent(heads=2, dim=16, rot_dim=16, vdim=16, window=44, scale=-0.3),
    "hgrn2": cases.hgrn2(),
    "hgrn2_odd": cases.hgrn2(heads=3, dim=7, vdim=5),
    "hgrn2_wide": cases.hgrn2(heads=1, dim=96, vdim=272),
    "hgrn2_large": cases.hgrn2(heads=2, dim=264, vdim=24),
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
    tol = TOL[dtype] * (2 if name.startswith("latent") and dtype is BF16 else 1)
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
            step = {r: 1 if at[r] >= decode_from else min(sizes[i % len(sizes)], lens[r] - at[r], max(decode_from - at[r], 1)) for r in rows}
            h = np.concatenate([x[r][at[r]:at[r] + step[r]] for r in rows])
            b = c.begin([step[r] for r in rows], rows)
            with torch.inference_mode():
                y = mix(on_gpu(h, dtype), b, c.arrays(0))[0].double().cpu().numpy()
            o = 0
            for r in rows:
                got[r][at[r]:at[r] + step[r]] = y[o:o + step[r]]
                o, at[r] = o + step[r], at[r] + step[r]
            i += 1
        c.check_status()
        for r in range(3):
            assert worst_row(got[r], want[r]) < tol and rel_rms(got[r], want[r]) < tol / 3, (sizes, decode_from, r)


@pytest.mark.parametrize("heads", [5, 20])
def test_decode_over_many_chunks_of_a_ring(heads):
    """A window of several split parts, sequences below, at and beyond it, prompt longer than the ring."""
    mix, oracle = _mixer(cases.latent(heads=heads, dim=40, rot_dim=24, vdim=72, kv_rank=136, window=700, scale=0.2), 48, 4, BF16)
    rng = np.random.default_rng(2)
    lens, tail = [1400, 702, 300, 260], 6
    x = [as_held(rng.standard_normal((n + tail, 48)), BF16) for n in lens]
    c = cache_of(mix.state(), dtype=BF16)
    c.open(4)
    with torch.inference_mode():
        mix(on_gpu(np.concatenate([a[:n] for a, n in zip(x, lens)]), BF16), c.begin(lens), c.arrays(0))
        got = [mix(on_gpu(np.stack([a[n + s] for a, n in zip(x, lens)]), BF16), c.begin(None), c.arrays(0))[0].double().cpu().numpy() for s in range(tail)]
    c.check_status()
    for r, (a, n) in enumerate(zip(x, lens)):
        assert worst_row(np.stack([g[r] for g in got]), oracle(a)[n:]) < 3e-2, r
