"""CPU restatement of the Dafovik decoder in float64 NumPy.  TEST INFRASTRUCTURE ONLY.

One function per mechanism, each a direct transcription of its defining equation: recurrences run token by token,
attention builds the full score matrix, nothing is cached or fused.  Nothing in the product package imports it and
it imports nothing from the product package.
"""
from __future__ import annotations

import numpy as np


def softplus(x):
    return np.maximum(x, 0.0) + np.log1p(np.exp(-np.abs(x)))


def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def unit_rms(x, eps):
    """x over its root mean square (last axis), eps under the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def post_norm_residual(x, y, w, mult, eps):
    """Residual update of a sublayer whose OUTPUT is normed."""
    return x + mult * centred_norm(y, w, eps)


def rotate_half_pairs(x, positions, base, dims):
    """x ``[T, heads, D]``: dimension i of the first ``dims`` turns with dimension i + dims/2."""
    half = dims // 2
    freq = np.power(float(base), -2.0 * np.arange(half) / dims)
    a = positions[:, None, None] * freq
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), rest], axis=-1)


def causal_conv_silu(x, w, bias):
    """x ``[T, C]``, w ``[C, taps]`` (last column: the current token), zeros before the start."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x], axis=0)
    y = np.zeros_like(x)
    for k in range(taps):
        y += w[:, k] * padded[k:k + x.shape[0]]
    return silu(y + bias)


def scalar_decay_recurrence(q, k, v, decay, state=None):
    """S_t = decay_t S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  q, k ``[T, H, N]``, v ``[T, H, P]``, decay ``[T, H]``.
    Returns ``(o [T, H, P], S [H, N, P])``."""
    T, H, N = q.shape
    S = np.zeros((H, N, v.shape[2])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnp,hn->hp", S, q[t])
    return o, S


def window_softmax(q, k, v, scale, window):
    """q ``[T, H, D]``, k ``[T, G, D]``, v ``[T, G, P]``: position i sees j with 0 <= i - j < window."""
    T, H, _ = q.shape
    G = k.shape[1]
    head = np.arange(H) // (H // G)
    s = np.einsum("ihd,jhd->hij", q, k[:, head]) * scale
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where((d >= 0) & (d < window), s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    p = p / p.sum(-1, keepdims=True)
    return np.einsum("hij,jhp->ihp", p, v[:, head])


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def differential_combine(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def grouped_gated_norm(y, z, w, groups, eps):
    """Gate first, then ``groups`` equal parts each over its own root mean square."""
    g = y * silu(z)
    T, C = g.shape
    return unit_rms(g.reshape(T, groups, C // groups), eps).reshape(T, C) * w


# ----------------------------------------------------------------------------------------------------- mixers
def mamba2_mixer(h, t, m, eps):
    """``t``: the mixer's tensors by name, ``m``: its sizes."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = h @ t["in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = causal_conv_silu(xbc, t["conv"], t["conv.b"])
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + t["dt_bias"])
    grp = np.arange(H) // (H // G)
    y, _ = scalar_decay_recurrence(C[:, grp], B[:, grp], dt[:, :, None] * x, np.exp(-np.exp(t["A_log"]) * dt))
    y = y + t["D"][:, None] * x
    y = grouped_gated_norm(y.reshape(T, inner), z, t["norm"], m["norm_groups"], eps)
    return y @ t["o"].T


def retention_mixer(h, t, m, eps):
    T = h.shape[0]
    H, D, P = m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=np.float64)
    q = rotate_half_pairs((h @ t["q"].T).reshape(T, H, D), pos, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_half_pairs((h @ t["k"].T).reshape(T, H, D), pos, m["rot"]["base"], m["rot"]["dims"]) * D ** -0.5
    v = (h @ t["v"].T).reshape(T, H, P)
    o, _ = scalar_decay_recurrence(q, k, v, np.tile(np.asarray(m["decay"], dtype=np.float64), (T, 1)))
    o = unit_rms(o, eps).reshape(T, H * P) * silu(h @ t["g"].T)
    return o @ t["o"].T


def differential_attention_mixer(h, t, m, eps):
    T = h.shape[0]
    H, G, D, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ t["q"].T).reshape(T, H, 2, D), eps) * t["q.norm"]
    k = unit_rms((h @ t["k"].T).reshape(T, G, 2, D), eps) * t["k.norm"]
    v = (h @ t["v"].T).reshape(T, G, P)
    a1 = window_softmax(q[:, :, 0], k[:, :, 0], v, m["scale"], m["mask"]["size"])
    a2 = window_softmax(q[:, :, 1], k[:, :, 1], v, m["scale"], m["mask"]["size"])
    lam = differential_lambda(t["lq1"], t["lk1"], t["lq2"], t["lk2"], m["diff"])
    o = differential_combine(a1, a2, lam, m["diff"], eps) * sigmoid(h @ t["g"].T)[:, :, None]
    return o.reshape(T, H * P) @ t["o"].T


MIXERS = {"mamba2": mamba2_mixer, "retention": retention_mixer, "attention": differential_attention_mixer}


def dense_mlp(h, up, down):
    return gelu_tanh(h @ up.T) @ down.T


def forward(cfg, tensors, ids, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence.  ``tensors``: name -> array; ``layers_out``: list that receives the
    residual stream after every layer."""
    t = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = t["embed"][np.asarray(ids)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in t.items() if k.startswith(p + "mix.")}
        y = MIXERS[layer["type"]](x, mix, layer["mixer"], eps)
        x = post_norm_residual(x, y, t[p + "norm1"], mult, eps)
        if layer.get("mlp") is not None:
            x = post_norm_residual(x, dense_mlp(x, t[p + "mlp.up"], t[p + "mlp.down"]), t[p + "norm2"], mult, eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return centred_norm(x, t["final.norm"], eps) @ t["head"].T
