"""Small configurations and random checkpoints for the tests of the latent-attention / HGRN2 decoder (error measures and the
checkpoint writer: ``dafovik_cases``)."""
import numpy as np
import torch


def latent(heads=3, dim=24, rot_dim=16, vdim=40, q_rank=56, kv_rank=48, window=19, scale=0.21, base=3000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                  "kv_rank": kv_rank, "mask": {"size": window}, "scale": scale,
                                                  "rot": {"base": base, "dims": rot_dim}}}


def hgrn2(heads=2, dim=24, vdim=40):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def experts(count=7, top=3, ff=40, identity=2, groups=(3, 2), scale=1.7):
    router = {"experts": count, "identity": identity, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def config(layers, width=72, vocab=151, groups=3, alpha=2.2, eps=3e-6, embed=1.9):
    """``layers``: (entry, feed-forward or None)."""
    return {"architecture": "Lonulix", "embedding": {"scale": embed}, "layers": [{**m, "mlp": f} for m, f in layers],
            "norm": {"eps": eps, "groups": groups}, "postln_alpha": alpha, "vocab": vocab, "width": width}


CONFIGS = {
    # every mixer and feed-forward, sizes that are multiples of 8 (the tensor-core kernels in bf16)
    "mixed": config([(hgrn2(), experts()), (latent(), dense()), (latent(window=7, heads=2, dim=72, vdim=72), experts(count=6, identity=0, groups=(2, 1), top=2)),
                     (hgrn2(heads=1, dim=72, vdim=16), None), (hgrn2(), dense(56))]),
    # odd sizes everywhere: scalar and token-by-token kernels, odd ranks, no groups of experts
    "odd": config([(latent(heads=3, dim=9, rot_dim=6, vdim=7, q_rank=13, kv_rank=11, window=11), experts(count=5, top=2, ff=13, identity=1, groups=None)),
                   (hgrn2(heads=3, dim=7, vdim=5), dense(41)), (hgrn2(heads=1, dim=10, vdim=9), experts(count=3, top=4, ff=9, identity=3, groups=(2, 2)))],
                  width=37, vocab=53, groups=1, alpha=1.0, embed=1.0),
    # sizes of one, a window of one, one expert, every expert chosen, heads beyond the tensor-core kernels, large ranks
    "extreme": config([(latent(heads=1, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=8, window=1), experts(count=1, top=1, ff=8, identity=0, groups=(1, 1), scale=1.0)),
                       (hgrn2(heads=1, dim=8, vdim=8), None),
                       (latent(heads=18, dim=136, rot_dim=72, vdim=136, q_rank=64, kv_rank=520, window=33, scale=0.06), experts(count=4, top=6, ff=16, identity=2, groups=(6, 6))),
                       (latent(heads=34, dim=16, rot_dim=2, vdim=8, q_rank=16, kv_rank=136, window=40), experts(count=8, top=1, ff=24, identity=0, groups=(4, 1)))],
                      width=48, vocab=64, groups=6, alpha=0.6, embed=0.5),
}


def random_tensors(cfg, seed=0, settled=False):
    """Checkpoint tensors (fp32 arrays holding bf16 values) with scales that keep every mechanism visible.  ``settled``: the
    corrections lie so far apart that they alone decide the choice of experts, which a rounding then cannot change."""
    rng = np.random.default_rng(seed)
    w = cfg["width"]

    def mat(o, i, s=1.0):
        return rng.standard_normal((o, i)) * s / np.sqrt(i)

    def vec(n, s=0.3, at=0.0):
        return at + s * rng.standard_normal(n)
    t = {"embed": rng.standard_normal((cfg["vocab"], w)), "final.norm": vec(w, at=1.0), "head": mat(cfg["vocab"], w)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        t.update({p + "norm1": vec(w, at=1.0), p + "rg1": mat(w, w), p + "rg1.b": vec(w, 0.5, 0.3)})
        if layer["type"] == "latent_attention":
            h, d, r, v, c, q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            t.update({p + "mix.dq": mat(q, w), p + "mix.dq.norm": vec(q, 0.3, 1.3), p + "mix.uq": mat(h * (d + r), q),
                      p + "mix.dkv": mat(c + r, w), p + "mix.dkv.norm": vec(c, 0.3, 1.2), p + "mix.uk": mat(h * d, c),
                      p + "mix.uv": mat(h * v, c), p + "mix.o": mat(w, h * v)})
        else:
            h, n, v = m["heads"], m["dim"], m["vdim"]
            t.update({p + "mix.q": mat(h * n, w), p + "mix.f": mat(h * n, w), p + "mix.f.b": vec(h * n, 2.0, 2.0),
                      p + "mix.lower": np.clip(vec(h * n, 0.3, 0.3), 0.0, 0.95), p + "mix.v": mat(h * v, w),
                      p + "mix.norm": vec(v, 0.3, 1.0), p + "mix.o": mat(w, h * v)})
        f = layer["mlp"]
        if f is None:
            continue
        t.update({p + "norm2": vec(w, at=1.0), p + "rg2": mat(w, w), p + "rg2.b": vec(w, 0.5, 0.3)})
        if f["kind"] == "dense":
            t.update({p + "mlp.gate": mat(f["ff"], w), p + "mlp.up": mat(f["ff"], w), p + "mlp.down": mat(w, f["ff"])})
        else:
            total = f["router"]["experts"] + f["router"]["identity"]
            t[p + "mlp.router"] = mat(total, w, 0.2 if settled else 1.0)
            t[p + "mlp.correction"] = rng.permutation(total) * 2.0 - total if settled else vec(total, 0.1, -1.5)   # below zero: a group that is
            for e in range(f["router"]["experts"]):                                                              # left out must not count as zero
                t.update({p + f"mlp.e{e}.up": mat(f["expert"]["ff"], w), p + f"mlp.e{e}.down": mat(w, f["expert"]["ff"])})
    return {k: torch.tensor(v, dtype=torch.float32).bfloat16().float().numpy() for k, v in t.items()}
