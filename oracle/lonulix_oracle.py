"""CPU restatement of the Lonulix decoder in float64 NumPy.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, each a direct transcription of its defining equation: the recurrence runs token by token,
attention builds every head's keys and the full score matrix, experts run one token at a time, nothing is cached, absorbed
or fused.  Nothing in the product package imports it and it imports nothing from the product package.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    e = np.exp(-np.abs(x))
    return np.where(x >= 0, 1.0, e) / (1.0 + e)


def silu(x):
    return x * sigmoid(x)


def gelu_erf(x):
    return 0.5 * x * (1.0 + np.vectorize(math.erf, otypes=[np.float64])(x / math.sqrt(2.0)))


def rms(x, w, eps):
    """Plain RMS norm over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def group_rms(x, w, groups, eps):
    """``groups`` equal consecutive parts, each over its own root mean square, then one weight for the whole vector."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, 1.0, eps).reshape(x.shape) * w


def gated_postnorm_residual(x, y, gate_w, gate_b, norm_w, alpha, groups, eps):
    """Norm of the sum; the sublayer's result is gated by its own input."""
    return group_rms(alpha * x + sigmoid(x @ gate_w.T + gate_b) * y, norm_w, groups, eps)


def rotate_neighbours(x, positions, base, dims):
    """x ``[T, ..., D]``: dimension 2i of the first ``dims`` turns with dimension 2i + 1."""
    x = x.copy()
    for i in range(dims // 2):
        a = positions * float(base) ** (-2.0 * i / dims)
        a = a.reshape(-1, *([1] * (x.ndim - 2)))
        u, v = x[..., 2 * i].copy(), x[..., 2 * i + 1].copy()
        x[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        x[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return x


def window_mask(T, window):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < window)


def two_part_attention(q_plain, q_turned, k_plain, k_turned, v, scale, window):
    """q_plain ``[T, H, D]``, q_turned ``[T, H, R]``, k_plain ``[T, H, D]``, k_turned ``[T, R]`` (all heads), v ``[T, H, P]``."""
    s = (np.einsum("ihd,jhd->hij", q_plain, k_plain) + np.einsum("ihr,jr->hij", q_turned, k_turned)) * scale
    s = np.where(window_mask(s.shape[1], window), s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("hij,jhp->ihp", p / p.sum(-1, keepdims=True), v)


def forget_gate(z, bias, lower):
    return lower + (1.0 - lower) * sigmoid(z + bias)


def channel_decay_recurrence(q, f, v, state=None):
    """S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, o_t = S_t^T q_t.  q, f ``[T, H, N]``, v ``[T, H, P]``.
    Returns ``(o [T, H, P], S [H, N, P])``."""
    T, H, N = q.shape
    S = np.zeros((H, N, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnp,hn->hp", S, q[t])
    return o, S


def route(z, correction, top, group_count, group_keep, scale):
    """Router logits of one token ``[E]`` -> ``(chosen experts, their weights)``: softmax scores, choice by corrected score
    among the experts of the best groups, weights from the scores without the correction."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    choice = s + correction
    size = len(z) // group_count
    best = choice.reshape(group_count, size).max(1)
    kept = np.argsort(-best, kind="stable")[:group_keep]
    open_ = np.full(len(z), -np.inf)
    for g in kept:
        open_[g * size:(g + 1) * size] = choice[g * size:(g + 1) * size]
    chosen = np.argsort(-open_, kind="stable")[:top]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20) * scale


# ----------------------------------------------------------------------------------------------------- sublayers
def latent_attention_mixer(h, t, m, eps):
    """``t``: the mixer's tensors by name, ``m``: its sizes."""
    T = h.shape[0]
    H, D, R, P, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T, dtype=np.float64)
    q = (rms(h @ t["dq"].T, t["dq.norm"], eps) @ t["uq"].T).reshape(T, H, D + R)
    down = h @ t["dkv"].T
    c = rms(down[:, :C], t["dkv.norm"], eps)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    k_turned = rotate_neighbours(down[:, C:], pos, base, dims)
    q_turned = rotate_neighbours(q[..., D:], pos, base, dims)
    k, v = (c @ t["uk"].T).reshape(T, H, D), (c @ t["uv"].T).reshape(T, H, P)
    o = two_part_attention(q[..., :D], q_turned, k, k_turned, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * P) @ t["o"].T


def hgrn2_mixer(h, t, m, eps):
    T = h.shape[0]
    H, N, P = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ t["q"].T).reshape(T, H, N)
    f = forget_gate(h @ t["f"].T, t["f.b"], t["lower"]).reshape(T, H, N)
    v = (h @ t["v"].T).reshape(T, H, P)
    o, _ = channel_decay_recurrence(q, f, v)
    return rms(o, t["norm"], eps).reshape(T, H * P) @ t["o"].T


MIXERS = {"latent_attention": latent_attention_mixer, "hgrn2": hgrn2_mixer}


def swiglu_mlp(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def expert_mlp(h, t, m):
    r = m["router"]
    real, same = r["experts"], r.get("identity", 0)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    y = np.zeros_like(h)
    for i, x in enumerate(h):
        chosen, w = route(t["router"] @ x, t["correction"], r["top"], groups["count"], groups["keep"], r["scale"])
        for e, g in zip(chosen, w):
            y[i] += g * (x if e >= real else t[f"e{e}.down"] @ gelu_erf(t[f"e{e}.up"] @ x))
    assert len(t["correction"]) == real + same
    return y


def feed_forward(h, t, m):
    return expert_mlp(h, t, m) if m["kind"] == "moe" else swiglu_mlp(h, t["gate"], t["up"], t["down"])


def forward(cfg, tensors, ids, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence.  ``tensors``: name -> array; ``layers_out``: list that receives the
    residual stream after every layer."""
    t = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps, groups, alpha = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["postln_alpha"]
    x = t["embed"][np.asarray(ids)] * cfg["embedding"]["scale"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in t.items() if k.startswith(prefix)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](x, sub(p + "mix."), layer["mixer"], eps)
        x = gated_postnorm_residual(x, y, t[p + "rg1"], t[p + "rg1.b"], t[p + "norm1"], alpha, groups, eps)
        if layer.get("mlp") is not None:
            y = feed_forward(x, sub(p + "mlp."), layer["mlp"])
            x = gated_postnorm_residual(x, y, t[p + "rg2"], t[p + "rg2.b"], t[p + "norm2"], alpha, groups, eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return group_rms(x, t["final.norm"], groups, eps) @ t["head"].T
