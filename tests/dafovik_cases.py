"""Small configurations, random checkpoints and error measures shared by the tests of the hybrid decoder."""
import json
import os

import numpy as np
import torch


def retention(heads=2, dim=16, vdim=24, rot=8, base=5000.0, decay=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                                           "decay": decay or [1 - 2.0 ** -(3 + 1.7 * i) for i in range(heads)]}}


def mamba2(heads=4, vdim=16, state=24, groups=2, conv=3, norm_groups=2):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def attention(heads=4, kv_heads=2, dim=24, vdim=40, window=19, scale=0.23, diff=0.35):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "mask": {"size": window}, "scale": scale, "diff": diff}}


def config(layers, width=72, vocab=151, ff=88, mult=0.7, eps=3e-6):
    """``layers``: entries of the functions above; a layer given as (entry, None) has no feed-forward."""
    out = []
    for layer in layers:
        entry, mlp = layer if isinstance(layer, tuple) else (layer, {"kind": "dense", "ff": ff})
        out.append({**entry, "mlp": mlp})
    return {"architecture": "Dafovik", "layers": out, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


CONFIGS = {
    # every mixer, sizes that are multiples of 8 (the tensor-core kernels in bf16)
    "mixed": config([mamba2(), attention(), retention(), (attention(window=7, heads=2, kv_heads=2), None), mamba2(conv=4)]),
    # odd sizes everywhere: scalar and token-by-token kernels
    "odd": config([retention(heads=3, dim=10, vdim=7, rot=6), attention(heads=3, kv_heads=1, dim=13, vdim=9, window=11),
                   mamba2(heads=3, vdim=5, state=9, groups=1, conv=2, norm_groups=3)], width=37, vocab=53, ff=41, mult=1.0),
    # sizes of one, a window of one, one tap, rotation of all dims, heads beyond 128
    "extreme": config([retention(heads=1, dim=8, vdim=8, rot=8, decay=[0.9]), mamba2(heads=2, vdim=8, state=8, groups=1, conv=1, norm_groups=1),
                       attention(heads=2, kv_heads=1, dim=8, vdim=8, window=1), attention(heads=1, kv_heads=1, dim=136, vdim=200, window=33)],
                      width=48, vocab=64, mult=0.4),
}


def random_tensors(cfg, seed=0):
    """Checkpoint tensors (fp32 arrays holding bf16 values) with scales that keep every mechanism visible."""
    rng = np.random.default_rng(seed)
    w = cfg["width"]

    def mat(o, i, s=1.0):
        return rng.standard_normal((o, i)) * s / np.sqrt(i)

    def vec(n, s=0.3, at=0.0):
        return at + s * rng.standard_normal(n)
    t = {"embed": rng.standard_normal((cfg["vocab"], w)), "final.norm": vec(w), "head": mat(cfg["vocab"], w)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"] = vec(w)
        if layer["type"] == "retention":
            h, d, v = m["heads"], m["dim"], m["vdim"]
            t.update({p + "mix.q": mat(h * d, w), p + "mix.k": mat(h * d, w), p + "mix.v": mat(h * v, w), p + "mix.g": mat(h * v, w),
                      p + "mix.o": mat(w, h * v)})
        elif layer["type"] == "mamba2":
            h, inner, ch = m["heads"], m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            t.update({p + "mix.in": mat(inner + ch + h, w), p + "mix.conv": vec((ch, m["conv"]), 0.6), p + "mix.conv.b": vec(ch),
                      p + "mix.dt_bias": vec(h, 0.5, -2.0), p + "mix.A_log": vec(h, 1.0, -1.0), p + "mix.D": vec(h, 0.5, 1.0),
                      p + "mix.norm": vec(inner, 0.3, 1.0), p + "mix.o": mat(w, inner)})
        else:
            h, g, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t.update({p + "mix.q": mat(2 * h * d, w), p + "mix.k": mat(2 * g * d, w), p + "mix.v": mat(g * v, w), p + "mix.g": mat(h, w),
                      p + "mix.q.norm": vec(d, 0.3, 1.5), p + "mix.k.norm": vec(d, 0.3, 1.5), p + "mix.o": mat(w, h * v),
                      **{p + f"mix.{n}": vec(d, 0.25) for n in ("lq1", "lk1", "lq2", "lk2")}})
        if layer["mlp"] is not None:
            t.update({p + "norm2": vec(w), p + "mlp.up": mat(layer["mlp"]["ff"], w), p + "mlp.down": mat(w, layer["mlp"]["ff"])})
    return {k: torch.tensor(v, dtype=torch.float32).bfloat16().float().numpy() for k, v in t.items()}


def write_checkpoint(path, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: torch.from_numpy(v).bfloat16().contiguous() for k, v in tensors.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def rel_rms(got, want):
    got = got.detach().double().cpu().numpy() if torch.is_tensor(got) else np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return float(np.sqrt(np.mean((got - want) ** 2)) / (np.sqrt(np.mean(want ** 2)) + 1e-30))


def worst_row(got, want):
    """Largest RMS difference of a row (first axis) relative to the RMS of that row, or of a middling row if that is larger:
    one wrong row does not average away, and one large row does not hide the others."""
    got = got.detach().double().cpu().numpy() if torch.is_tensor(got) else np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    axes = tuple(range(1, got.ndim))
    size = np.sqrt(np.mean(want ** 2, axis=axes))
    return float((np.sqrt(np.mean((got - want) ** 2, axis=axes)) / (np.maximum(size, np.median(size)) + 1e-30)).max())
