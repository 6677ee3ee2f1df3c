"""Lonulix: a hybrid decoder of windowed latent-attention and HGRN2 layers with dense or expert feed-forwards.

The order of layers, each layer's mixer and feed-forward and all sizes and constants come from the configuration.  The norm
comes after the sum, in groups, and a sublayer's result is gated by the sublayer's own input:

    x <- norm1(alpha x + sigmoid(G1 x + b1) * mixer(x)),   x <- norm2(alpha x + sigmoid(G2 x + b2) * ff(x)).

The gate's product is part of the sublayer's fused projection; gate, sum, norm and (for experts) the gathering of the expert
rows are one kernel.  Everything else is that of the hybrid decoders (``modeling_hybrid``).
"""
from __future__ import annotations

from typing import List, Optional

import torch
from torch import nn

from . import ops
from .feedforward import RoutedSum, SparseMLP, SwiGLU
from .mixers import HGRN2Mixer, LatentAttentionMixer, as_f32
from .modeling_hybrid import HybridConfig, HybridForCausalLM, HybridModel, StreamNorm
from .state_cache import StepBatch


def _latent_attention(width, m, eps):
    return LatentAttentionMixer(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["mask"]["size"],
                                m["scale"], m["rot"]["dims"], m["rot"]["base"], eps, gate_rows=width)


def _hgrn2(width, m, eps):
    return HGRN2Mixer(width, m["heads"], m["dim"], m["vdim"], eps, gate_rows=width)


def _dense(width, m):
    return SwiGLU(width, m["ff"], gate_rows=width)


def _experts(width, m):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return SparseMLP(width, m["expert"]["ff"], r["experts"], r["top"], r.get("scale", 1.0), r.get("identity", 0) or 0, groups["count"],
                     groups["keep"], gate_rows=width)


MIXERS = {"latent_attention": _latent_attention, "hgrn2": _hgrn2}
FEED_FORWARDS = {"dense": _dense, "moe": _experts}


class LonulixConfig(HybridConfig):
    """``mlp``: {"kind": "dense", "ff": n}, {"kind": "moe", "expert": {"ff": n}, "router": {...}} or None; ``embedding.scale``,
    ``norm.groups`` and ``postln_alpha`` beside the entries of ``HybridConfig``."""

    model_type = "lonulix"
    architecture = "Lonulix"
    mixers = MIXERS
    feed_forwards = FEED_FORWARDS
    checkpoint_keys = ("embedding", "layers", "norm", "postln_alpha", "vocab", "width")

    def __init__(self, layers: Optional[List[dict]] = None, norm: Optional[dict] = None, embedding: Optional[dict] = None,
                 postln_alpha: float = 1.0, vocab: int = 256, width: int = 64, **kwargs):
        self.embedding = dict(embedding or {"scale": 1.0})
        self.postln_alpha = float(postln_alpha)
        super().__init__(layers, norm, vocab, width, **kwargs)
        self.norm.setdefault("groups", 1)
        if self.width % self.norm["groups"]:
            raise ValueError(f"a width of {self.width} in {self.norm['groups']} norm groups")


class LonulixLayer(nn.Module):
    def __init__(self, config: LonulixConfig, idx: int):
        super().__init__()
        spec, width = config.layers[idx], config.width
        self.eps, self.groups, self.alpha = float(config.norm["eps"]), int(config.norm["groups"]), config.postln_alpha
        self.mix = MIXERS[spec["type"]](width, spec["mixer"], self.eps)
        self.norm1, self.gate1_bias = StreamNorm(width), nn.Parameter(torch.zeros(width))
        self.mlp = self.norm2 = None
        if spec.get("mlp") is not None:
            self.mlp = FEED_FORWARDS[spec["mlp"].get("kind", "dense")](width, spec["mlp"])
            self.norm2, self.gate2_bias = StreamNorm(width), nn.Parameter(torch.zeros(width))

    def checkpoint(self):
        out = {"norm1": self.norm1.weight, "rg1": self.mix.gate_part(), "rg1.b": self.gate1_bias,
               **{f"mix.{k}": v for k, v in self.mix.checkpoint().items()}}
        if self.mlp is not None:
            out.update({"norm2": self.norm2.weight, "rg2": self.mlp.gate_part(), "rg2.b": self.gate2_bias,
                        **{f"mlp.{k}": v for k, v in self.mlp.checkpoint().items()}})
        return out

    def reset_parameters(self, std: float) -> None:
        nn.init.zeros_(self.gate1_bias)
        if self.mlp is not None:
            nn.init.zeros_(self.gate2_bias)

    def _close(self, stream, copy, result, norm, bias):
        y, gate = result
        routed = {}
        if isinstance(y, RoutedSum):
            routed, y = dict(place=y.place, choice_weight=y.weight), y.rows
        ops.gated_sum_norm(stream, y, as_f32(norm, "weight"), copy, self.groups, self.eps, self.alpha, gate, as_f32(self, bias), **routed)

    def forward(self, stream: torch.Tensor, copy: Optional[torch.Tensor], batch: StepBatch, data: dict) -> None:
        """Updates the fp32 stream and its copy in the model type (None: the stream is in the model type) in place."""
        x = stream if copy is None else copy
        self._close(stream, copy, self.mix(x, batch, data), self.norm1, "gate1_bias")
        if self.mlp is not None:
            self._close(stream, copy, self.mlp(x, batch.status), self.norm2, "gate2_bias")


class LonulixModel(HybridModel):
    config_class = LonulixConfig
    _no_split_modules = ["LonulixLayer"]
    layer_cls = LonulixLayer

    def __init__(self, config: LonulixConfig):
        self.embed_scale, self.norm_groups = float(config.embedding["scale"]), int(config.norm["groups"])
        super().__init__(config)


class LonulixForCausalLM(HybridForCausalLM):
    config_class = LonulixConfig
    _no_split_modules = ["LonulixLayer"]
    model_cls = LonulixModel


__all__ = ["LonulixConfig", "LonulixForCausalLM", "LonulixModel"]
