"""Feed-forward layers of hybrid decoders beside ``mixers.GeluMLP``: a gated dense one and a mixture of experts.

Like a mixer, a feed-forward built with ``gate_rows`` also computes that many rows of a gate of its input (``gate_part()`` is
their weight) and returns ``(result, gate logits)``.  Sizes and constants are constructor arguments.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch
import torch.nn.functional as F
from torch import nn

from . import ops
from .mixers import FusedProjection, as_f32


@dataclass
class RoutedSum:
    """A result that is still to be added up: of token t the sum over c of ``weight[t, c] * rows[place[t, c]]``, the layer's
    own input standing where ``place`` is -1."""
    rows: torch.Tensor
    place: torch.Tensor
    weight: torch.Tensor


class FeedForward(nn.Module):
    gate_rows = 0

    def checkpoint(self) -> Dict[str, torch.Tensor]:
        raise NotImplementedError

    def gate_part(self) -> torch.Tensor:
        return self.proj.part("gate_rows")

    def reset_parameters(self, std: float) -> None:
        raise NotImplementedError

    def _gate(self, u: torch.Tensor) -> torch.Tensor:
        lo, hi = self.proj.offsets["gate_rows"]
        return u[:, lo:hi]


class SwiGLU(FeedForward):
    """``W_down (silu(W_gate h) * (W_up h))``; gate, up and the gate rows are one product."""

    def __init__(self, width: int, ff: int, gate_rows: int = 0):
        super().__init__()
        self.ff, self.gate_rows = ff, gate_rows
        self.proj = FusedProjection(width, {"gate": ff, "up": ff, "gate_rows": gate_rows})
        self.down = nn.Parameter(torch.zeros(width, ff))

    def checkpoint(self):
        return {"gate": self.proj.part("gate"), "up": self.proj.part("up"), "down": self.down}

    def reset_parameters(self, std):
        self.proj.reset_parameters(std)
        nn.init.normal_(self.down, mean=0.0, std=std)

    def forward(self, x, status=None):
        u = self.proj(x)
        act = torch.empty(x.shape[0], self.ff, dtype=x.dtype, device=x.device)
        ops.swiglu(u, act)
        y = F.linear(act, self.down)
        return (y, self._gate(u)) if self.gate_rows else y


class SparseMLP(FeedForward):
    """Mixture of experts ``W_down gelu(W_up h)`` (erf form) with softmax scores, a correction that counts for the choice only,
    group-limited choice and ``identity`` experts that return their input.  The result is a ``RoutedSum``."""

    def __init__(self, width: int, ff: int, experts: int, top: int, scale: float = 1.0, identity: int = 0, groups: int = 1,
                 keep: int = 1, gate_rows: int = 0):
        super().__init__()
        if (experts + identity) % groups or not 0 < keep <= groups or not 0 < top <= keep * ((experts + identity) // groups):
            raise ValueError(f"{top} of {experts} + {identity} experts in {groups} groups, {keep} kept")
        self.experts, self.top, self.scale, self.identity = experts, top, float(scale), identity
        self.groups, self.keep, self.gate_rows = groups, keep, gate_rows
        self.up = nn.Parameter(torch.zeros(experts, ff, width))
        self.down = nn.Parameter(torch.zeros(experts, width, ff))
        self.router = nn.Parameter(torch.zeros(experts + identity, width))
        self.correction = nn.Parameter(torch.zeros(experts + identity))
        if gate_rows:
            self.proj = FusedProjection(width, {"gate_rows": gate_rows})

    def checkpoint(self):
        out = {"router": self.router, "correction": self.correction}
        for e in range(self.experts):
            out[f"e{e}.up"], out[f"e{e}.down"] = self.up[e], self.down[e]
        return out

    def reset_parameters(self, std):
        for w in (self.up, self.down, self.router):
            nn.init.normal_(w, mean=0.0, std=std)
        nn.init.zeros_(self.correction)
        if self.gate_rows:
            self.proj.reset_parameters(std)

    def route(self, x):
        """Router logits in fp32, then ``(place, weight, src, offsets)``."""
        z = F.linear(x, self.router) if x.dtype == torch.float32 else torch.mm(x, self.router.t(), out_dtype=torch.float32)
        return ops.moe_route(z, as_f32(self, "correction"), self.identity, self.top, self.groups, self.keep, self.scale)

    def forward(self, x, status: Optional[torch.Tensor] = None):
        place, weight, src, offsets = self.route(x)
        hidden = torch.empty(src.shape[0], self.up.shape[1], dtype=x.dtype, device=x.device)
        ops.moe_gemm(x, self.up, offsets, hidden, src=src, act="gelu", status=status)
        rows = torch.empty(src.shape[0], x.shape[1], dtype=x.dtype, device=x.device)
        ops.moe_gemm(hidden, self.down, offsets, rows, status=status)
        y = RoutedSum(rows, place, weight)
        return (y, self._gate(self.proj(x))) if self.gate_rows else y


__all__ = ["FeedForward", "RoutedSum", "SparseMLP", "SwiGLU"]
