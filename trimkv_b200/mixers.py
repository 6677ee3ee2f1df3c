"""Token mixers of hybrid decoders: retention, state-space duality (Mamba-2), HGRN2, windowed differential attention and
windowed latent attention.

A mixer reads the packed tokens of a step, keeps its requests' state in ``HybridStateCache`` slots and runs the CUDA
kernels: one fused projection, the mixing kernels (a chunked or windowed form for steps of several tokens, a one-token form
for decoding), and the output projection.  Sizes and constants are constructor arguments; a mixer knows nothing of the
design it is part of.  Small weight vectors reach the kernels as fp32 (``as_f32``).
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch
import torch.nn.functional as F
from torch import nn

from . import ops
from .state_cache import LatentState, RecurrentState, StepBatch, WindowState


def _stamp(p: torch.Tensor):
    """Changes when the tensor is written in place or replaced (tensors made in inference mode keep no version)."""
    return (p.data_ptr(), 0 if p.is_inference() else p._version, p.dtype, p.device)


def as_f32(module: nn.Module, name: str) -> torch.Tensor:
    """The parameter as a contiguous fp32 array; the converted copy is kept until the parameter changes or moves."""
    p = getattr(module, name)
    if p.dtype == torch.float32 and p.is_contiguous():
        return p.detach()
    memo = module.__dict__.setdefault("_f32", {})
    key = _stamp(p)
    hit = memo.get(name)
    if hit is None or hit[0] != key:
        hit = (key, p.detach().float().contiguous())
        memo[name] = hit
    return hit[1]


class FusedProjection(nn.Module):
    """One weight for several linear maps of the same input, rows in the order given, padded with zero rows so that a row
    of the output starts on a 16-byte boundary."""

    def __init__(self, width: int, parts: Dict[str, int]):
        super().__init__()
        self.offsets, at = {}, 0
        for name, rows in parts.items():
            self.offsets[name] = (at, at + rows)
            at += rows
        self.used = at
        self.weight = nn.Parameter(torch.zeros(-(-at // 8) * 8, width))

    def part(self, name: str) -> torch.Tensor:
        lo, hi = self.offsets[name]
        return self.weight[lo:hi]

    def reset_parameters(self, std: float) -> None:
        nn.init.normal_(self.weight, mean=0.0, std=std)
        with torch.no_grad():
            self.weight[self.used:].zero_()

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return F.linear(x, self.weight)


def rotary_frequencies(base: float, dims: int) -> torch.Tensor:
    """``base^(-2i/dims)`` for the pairs i, each as a high and a low fp32 part ``[dims / 2, 2]``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / max(dims, 1))
    hi = f.float()
    return torch.stack([hi, (f - hi.double()).float()], dim=1).contiguous()


class Mixer(nn.Module):
    """``state()`` describes what a request keeps; ``checkpoint()`` maps the names a checkpoint uses to parameters.

    Mixers built with ``gate_rows`` compute that many rows of a gate of the same input in their fused projection:
    ``gate_part()`` is its weight, and ``forward`` returns ``(result, gate logits)``."""

    gate_rows = 0

    def gate_part(self) -> torch.Tensor:
        return self.proj.part("gate_rows")

    def _gate(self, u: torch.Tensor) -> torch.Tensor:
        lo, hi = self.proj.offsets["gate_rows"]
        return u[:, lo:hi]

    def state(self):
        raise NotImplementedError

    def checkpoint(self) -> Dict[str, torch.Tensor]:
        raise NotImplementedError

    def reset_parameters(self, std: float) -> None:
        raise NotImplementedError

    def forward(self, x: torch.Tensor, batch: StepBatch, data: dict) -> torch.Tensor:
        raise NotImplementedError

    def _constant(self, key, device, make) -> torch.Tensor:
        """An fp32 table that depends on the configuration only, built once per device (never cast with the model)."""
        memo = self.__dict__.setdefault("_tables", {})
        t = memo.get((key, device))
        if t is None:
            t = memo[(key, device)] = make().to(device)
        return t


class RetentionMixer(Mixer):
    """Linear attention with a fixed decay per head, rotary q and k, a per-head RMS norm and a SiLU gate."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay, rot_dims: int, rot_base: float, eps: float):
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        if rot_dims % 2 or rot_dims > dim:
            raise ValueError(f"rotary dims {rot_dims} of a head of {dim}")
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.decay, self.rot_dims, self.rot_base = [float(d) for d in decay], rot_dims, float(rot_base)
        self.proj = FusedProjection(width, {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim})
        self.o = nn.Parameter(torch.zeros(width, heads * vdim))

    def state(self):
        return RecurrentState(self.heads, self.dim, self.vdim)

    def checkpoint(self):
        return {**{n: self.proj.part(n) for n in ("q", "k", "v", "g")}, "o": self.o}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        nn.init.normal_(self.o, mean=0.0, std=std)

    def _freq(self, device):
        return self._constant("freq", device, lambda: rotary_frequencies(self.rot_base, self.rot_dims))

    def _decay(self, device, log: bool):
        return self._constant(("decay", log), device, lambda: (
            torch.tensor([math.log(d) if d > 0 else -1e30 for d in self.decay] if log else self.decay,
                         dtype=torch.float64).float()))

    def forward(self, x, batch, data):
        h, d, p = self.heads, self.dim, self.vdim
        u = self.proj(x)
        out = torch.empty(x.shape[0], h * p, dtype=x.dtype, device=x.device)
        freq = self._freq(x.device)
        if batch.cu is None:
            ops.retention_step(u, data["state"], batch, self._decay(x.device, False), freq, out, d, self.rot_dims, d ** -0.5, self.eps)
            return F.linear(out, self.o)
        qk = torch.empty(x.shape[0], 2 * h * d, dtype=x.dtype, device=x.device)
        ops.rotate_qk(u, qk, batch, h, d, self.rot_dims, freq, d ** -0.5)
        y = torch.empty_like(out)
        ops.linrec(qk[:, :h * d], qk[:, h * d:], u[:, 2 * h * d:2 * h * d + h * p], data["state"], batch, y, h,
                   head_decay=self._decay(x.device, False), head_log_decay=self._decay(x.device, True))
        ops.gated_norm(y, u[:, 2 * h * d + h * p:2 * h * (d + p)], None, out, h, self.eps, gate_first=False)
        return F.linear(out, self.o)


class SSDMixer(Mixer):
    """State-space duality: input-dependent decay per head, B and C shared by the heads of a group, short convolution."""

    def __init__(self, width: int, heads: int, vdim: int, state: int, groups: int, taps: int, norm_groups: int, eps: float):
        super().__init__()
        if heads % groups or (heads * vdim) % norm_groups:
            raise ValueError(f"{heads} heads in {groups} groups, {heads * vdim} channels in {norm_groups} norm groups")
        self.heads, self.vdim, self.n, self.groups = heads, vdim, state, groups
        self.taps, self.norm_groups, self.eps = taps, norm_groups, eps
        self.inner = heads * vdim
        self.channels = self.inner + 2 * groups * state
        self.proj = FusedProjection(width, {"in": self.inner + self.channels + heads})
        self.conv = nn.Parameter(torch.zeros(self.channels, taps))
        self.conv_bias = nn.Parameter(torch.zeros(self.channels))
        self.dt_bias = nn.Parameter(torch.zeros(heads))
        self.a_log = nn.Parameter(torch.zeros(heads))
        self.skip = nn.Parameter(torch.ones(heads))
        self.norm = nn.Parameter(torch.ones(self.inner))
        self.o = nn.Parameter(torch.zeros(width, self.inner))

    def state(self):
        return RecurrentState(self.heads, self.n, self.vdim, self.taps, self.channels)

    def checkpoint(self):
        return {"in": self.proj.part("in"), "conv": self.conv, "conv.b": self.conv_bias, "dt_bias": self.dt_bias,
                "A_log": self.a_log, "D": self.skip, "norm": self.norm, "o": self.o}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        nn.init.normal_(self.o, mean=0.0, std=std)
        with torch.no_grad():
            nn.init.uniform_(self.conv, -self.taps ** -0.5, self.taps ** -0.5)
            nn.init.zeros_(self.conv_bias)
            nn.init.ones_(self.skip)
            nn.init.ones_(self.norm)
            nn.init.uniform_(self.a_log, 0.0, math.log(16.0))
            dt = torch.exp(torch.empty_like(self.dt_bias, dtype=torch.float32).uniform_(math.log(1e-3), math.log(1e-1)))
            self.dt_bias.copy_(dt + torch.log(-torch.expm1(-dt)))     # softplus(dt_bias) = dt

    def forward(self, x, batch, data):
        inner, ch, h, gn = self.inner, self.channels, self.heads, self.groups * self.n
        u = self.proj(x)
        y = torch.empty(x.shape[0], inner, dtype=x.dtype, device=x.device)
        w, b, dtb, a_log, skip = (as_f32(self, n) for n in ("conv", "conv_bias", "dt_bias", "a_log", "skip"))
        if batch.cu is None:
            ops.ssd_step(u, data["conv"], data["state"], batch, w, b, dtb, a_log, skip, y, self.groups)
        else:
            xbc = torch.empty(x.shape[0], ch, dtype=x.dtype, device=x.device)
            ops.conv_silu(u[:, inner:inner + ch], data["conv"], w, b, xbc, batch)
            dt = torch.empty(x.shape[0], h, dtype=torch.float32, device=x.device)
            log_decay = torch.empty_like(dt)
            ops.ssd_steps(u[:, inner + ch:inner + ch + h], dtb, a_log, dt, log_decay)
            ops.linrec(xbc[:, inner + gn:], xbc[:, inner:inner + gn], xbc[:, :inner], data["state"], batch, y, self.groups,
                       log_decay=log_decay, v_scale=dt, skip=skip)
        out = torch.empty_like(y)
        ops.gated_norm(y, u[:, :inner], as_f32(self, "norm"), out, self.norm_groups, self.eps, gate_first=True)
        return F.linear(out, self.o)


class DifferentialAttentionMixer(Mixer):
    """Two softmax maps over the same values inside a sliding window, without positions; q and k normed per head and map,
    the difference of the maps normed per head, one output gate per head."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int, scale: float, diff: float, eps: float):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads on {kv_heads} key/value heads")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.window, self.scale, self.diff, self.eps = window, float(scale), float(diff), eps
        self.proj = FusedProjection(width, {"q": heads * 2 * dim, "k": kv_heads * 2 * dim, "v": kv_heads * vdim, "g": heads})
        self.q_norm = nn.Parameter(torch.ones(dim))
        self.k_norm = nn.Parameter(torch.ones(dim))
        self.lq1, self.lk1 = nn.Parameter(torch.zeros(dim)), nn.Parameter(torch.zeros(dim))
        self.lq2, self.lk2 = nn.Parameter(torch.zeros(dim)), nn.Parameter(torch.zeros(dim))
        self.o = nn.Parameter(torch.zeros(width, heads * vdim))

    def state(self):
        return WindowState(self.kv_heads, -(-self.dim // 64) * 64, -(-self.vdim // 64) * 64, self.window)

    def checkpoint(self):
        return {**{n: self.proj.part(n) for n in ("q", "k", "v", "g")}, "q.norm": self.q_norm, "k.norm": self.k_norm,
                "lq1": self.lq1, "lk1": self.lk1, "lq2": self.lq2, "lk2": self.lk2, "o": self.o}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        nn.init.normal_(self.o, mean=0.0, std=std)
        for w in (self.q_norm, self.k_norm):
            nn.init.ones_(w)
        for w in (self.lq1, self.lk1, self.lq2, self.lk2):
            nn.init.normal_(w, mean=0.0, std=0.1)

    def _lambda(self) -> torch.Tensor:
        """``exp(lq1 . lk1) - exp(lq2 . lk2) + diff`` on the device, recomputed when one of the vectors changes."""
        vecs = (self.lq1, self.lk1, self.lq2, self.lk2)
        key = tuple(_stamp(v) for v in vecs)
        memo = self.__dict__.get("_lam")
        if memo is None or memo[0] != key:
            a, b, c, d = (v.detach().float() for v in vecs)
            memo = self.__dict__["_lam"] = (key, (torch.exp((a * b).sum()) - torch.exp((c * d).sum()) + self.diff).reshape(1))
        return memo[1]

    def forward(self, x, batch, data):
        u = self.proj(x)
        out = torch.empty(x.shape[0], self.heads * self.vdim, dtype=x.dtype, device=x.device)
        g0, g1 = self.proj.offsets["g"]
        ops.diff_attention(u, u[:, g0:g1], as_f32(self, "q_norm"), as_f32(self, "k_norm"), data["k"], data["v"], batch,
                           self._lambda(), self.diff, self.scale, self.eps, out, self.heads, self.dim, self.vdim, self.window)
        return F.linear(out, self.o)


class HGRN2Mixer(Mixer):
    """Linear attention whose forget gate, one per head and channel and bounded from below, also decides what is written."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, eps: float, gate_rows: int = 0):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps, self.gate_rows = heads, dim, vdim, eps, gate_rows
        self.proj = FusedProjection(width, {"q": heads * dim, "f": heads * dim, "v": heads * vdim, "gate_rows": gate_rows})
        self.f_bias = nn.Parameter(torch.zeros(heads * dim))
        self.lower = nn.Parameter(torch.zeros(heads * dim))
        self.norm = nn.Parameter(torch.ones(vdim))
        self.o = nn.Parameter(torch.zeros(width, heads * vdim))

    def state(self):
        return RecurrentState(self.heads, self.dim, self.vdim)

    def checkpoint(self):
        return {**{n: self.proj.part(n) for n in ("q", "f", "v")}, "f.b": self.f_bias, "lower": self.lower, "norm": self.norm, "o": self.o}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        nn.init.normal_(self.o, mean=0.0, std=std)
        nn.init.ones_(self.norm)
        with torch.no_grad():
            self.f_bias.uniform_(0.0, 4.0)
            self.lower.uniform_(0.0, 0.5)

    def forward(self, x, batch, data):
        h, n, p = self.heads, self.dim, self.vdim
        u = self.proj(x)
        q, f, v = (u[:, lo:hi] for lo, hi in (self.proj.offsets[k] for k in ("q", "f", "v")))
        bias, lower, norm = (as_f32(self, k) for k in ("f_bias", "lower", "norm"))
        out = torch.empty(x.shape[0], h * p, dtype=x.dtype, device=x.device)
        if batch.cu is None:
            ops.chanrec_step(q, f, v, bias, lower, norm, data["state"], batch, out, self.eps)
        else:
            y = torch.empty_like(out)
            ops.chanrec(q, f, v, bias, lower, data["state"], batch, y)
            ops.gated_norm(y, None, norm, out, h, self.eps)
        y = F.linear(out, self.o)
        return (y, self._gate(u)) if self.gate_rows else y


class LatentAttentionMixer(Mixer):
    """Softmax attention inside a sliding window whose keys and values come from one normed latent per position; a rotated key
    part is shared by the heads.  A request keeps the latent and the rotated part only.

    Steps of several tokens expand the latents to every head's keys and values; one-token steps take the queries into the
    latent space instead (``W_uk`` on the query, ``W_uv`` on the weighted latents)."""

    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, window: int,
                 scale: float, rot_dims: int, rot_base: float, eps: float, gate_rows: int = 0):
        super().__init__()
        if rot_dims % 2 or rot_dims > rot_dim:
            raise ValueError(f"rotary dims {rot_dims} of a part of {rot_dim}")
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.window, self.scale, self.eps, self.gate_rows = window, float(scale), eps, gate_rows
        self.rot_dims, self.rot_base = rot_dims, float(rot_base)
        self.proj = FusedProjection(width, {"dq": q_rank, "dkv": kv_rank + rot_dim, "gate_rows": gate_rows})
        self.q_norm, self.kv_norm = nn.Parameter(torch.ones(q_rank)), nn.Parameter(torch.ones(kv_rank))
        self.uq = nn.Parameter(torch.zeros(heads * (dim + rot_dim), q_rank))
        self.ukv = FusedProjection(kv_rank, {"uk": heads * dim, "uv": heads * vdim})
        self.o = nn.Parameter(torch.zeros(width, heads * vdim))

    def state(self):
        return LatentState(-(-self.kv_rank // 64) * 64 + -(-self.rot_dim // 64) * 64, self.window)

    def checkpoint(self):
        return {"dq": self.proj.part("dq"), "dq.norm": self.q_norm, "uq": self.uq, "dkv": self.proj.part("dkv"),
                "dkv.norm": self.kv_norm, "uk": self.ukv.part("uk"), "uv": self.ukv.part("uv"), "o": self.o}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        self.ukv.reset_parameters(std)
        for w in (self.uq, self.o):
            nn.init.normal_(w, mean=0.0, std=std)
        for w in (self.q_norm, self.kv_norm):
            nn.init.ones_(w)

    def _freq(self, device):
        return self._constant("freq", device, lambda: rotary_frequencies(self.rot_base, self.rot_dims))

    def forward(self, x, batch, data):
        h, d, r, p, rank, T = self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, x.shape[0]
        u, freq = self.proj(x), self._freq(x.device)
        cq, lin = ops.latent_prep(u, as_f32(self, "q_norm"), as_f32(self, "kv_norm"), self.eps, r, self.rot_dims, freq, data["latent"],
                                  batch, self.window)
        q = F.linear(cq, self.uq)
        out = torch.empty(T, h * p, dtype=x.dtype, device=x.device)
        if batch.cu is None:
            q3 = q.view(T, h, d + r)
            q_abs = torch.bmm(q3[:, :, :d].transpose(0, 1), self.ukv.part("uk").view(h, d, rank))
            o_lat = torch.empty_like(q_abs)
            ops.latent_decode(q_abs.transpose(0, 1), q3, r, freq, data["latent"], batch, self.scale, o_lat.transpose(0, 1), self.rot_dims)
            torch.bmm(o_lat, self.ukv.part("uv").view(h, p, rank).transpose(1, 2), out=out.view(T, h, p).transpose(0, 1))
        else:
            ops.rotate_pairs(q, batch, h, d + r, d, self.rot_dims, freq)
            kv = self.ukv(lin[:, :rank])
            ops.latent_prefill(q, kv, lin, batch, self.scale, out, h, d, r, p, rank, self.window)
        y = F.linear(out, self.o)
        return (y, self._gate(u)) if self.gate_rows else y


class GeluMLP(nn.Module):
    """Dense feed-forward with the tanh form of GELU."""

    def __init__(self, width: int, ff: int):
        super().__init__()
        self.up = nn.Parameter(torch.zeros(ff, width))
        self.down = nn.Parameter(torch.zeros(width, ff))

    def checkpoint(self):
        return {"up": self.up, "down": self.down}

    def reset_parameters(self, std):
        nn.init.normal_(self.up, mean=0.0, std=std)
        nn.init.normal_(self.down, mean=0.0, std=std)

    def forward(self, x):
        u = F.linear(x, self.up)
        ops.gelu_tanh(u)
        return F.linear(u, self.down)


__all__ = ["DifferentialAttentionMixer", "FusedProjection", "GeluMLP", "HGRN2Mixer", "LatentAttentionMixer", "Mixer",
           "RetentionMixer", "SSDMixer", "as_f32", "rotary_frequencies"]
