"""Dafovik: a hybrid decoder of retention, state-space (Mamba-2) and windowed differential-attention layers.

The order of layers, each layer's mixer and all its sizes come from the configuration.  A sublayer reads the residual
stream itself and only its output is normed:  x <- x + m norm1(mixer(x)),  x <- x + m norm2(mlp(x)),  with RMS norms whose
weights are stored around zero.  Everything else is that of the hybrid decoders (``modeling_hybrid``).
"""
from __future__ import annotations

from typing import List, Optional

import torch
from torch import nn

from . import ops
from .mixers import DifferentialAttentionMixer, GeluMLP, Mixer, RetentionMixer, SSDMixer, as_f32
from .modeling_hybrid import HybridConfig, HybridForCausalLM, HybridModel, StreamNorm
from .state_cache import StepBatch


def _retention(width, m, eps):
    return RetentionMixer(width, m["heads"], m["dim"], m["vdim"], m["decay"], m["rot"]["dims"], m["rot"]["base"], eps)


def _mamba2(width, m, eps):
    return SSDMixer(width, m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"], eps)


def _attention(width, m, eps):
    return DifferentialAttentionMixer(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"],
                                      m["diff"], eps)


MIXERS = {"retention": _retention, "mamba2": _mamba2, "attention": _attention}


class DafovikConfig(HybridConfig):
    """``mlp``: {"kind": "dense", "ff": n} or None; ``residual_mult`` beside the entries of ``HybridConfig``."""

    model_type = "dafovik"
    architecture = "Dafovik"
    mixers = MIXERS
    feed_forwards = {"dense": GeluMLP}
    checkpoint_keys = ("layers", "norm", "residual_mult", "vocab", "width")

    def __init__(self, layers: Optional[List[dict]] = None, norm: Optional[dict] = None, residual_mult: float = 1.0,
                 vocab: int = 256, width: int = 64, **kwargs):
        self.residual_mult = float(residual_mult)
        super().__init__(layers, norm, vocab, width, **kwargs)


class DafovikLayer(nn.Module):
    def __init__(self, config: DafovikConfig, idx: int):
        super().__init__()
        spec = config.layers[idx]
        self.eps, self.mult = float(config.norm["eps"]), config.residual_mult
        self.mix: Mixer = MIXERS[spec["type"]](config.width, spec["mixer"], self.eps)
        self.norm1 = StreamNorm(config.width, centre=0.0)
        self.mlp = GeluMLP(config.width, spec["mlp"]["ff"]) if spec.get("mlp") is not None else None
        self.norm2 = StreamNorm(config.width, centre=0.0) if self.mlp is not None else None

    def checkpoint(self):
        out = {"norm1": self.norm1.weight, **{f"mix.{k}": v for k, v in self.mix.checkpoint().items()}}
        if self.mlp is not None:
            out.update({"norm2": self.norm2.weight, **{f"mlp.{k}": v for k, v in self.mlp.checkpoint().items()}})
        return out

    def forward(self, stream: torch.Tensor, copy: Optional[torch.Tensor], batch: StepBatch, data: dict) -> None:
        """Updates the fp32 stream and its copy in the model type (None: the stream is in the model type) in place."""
        x = stream if copy is None else copy
        ops.postnorm_add(stream, self.mix(x, batch, data), as_f32(self.norm1, "weight"), copy, self.eps, self.mult, 1.0)
        if self.mlp is not None:
            ops.postnorm_add(stream, self.mlp(x), as_f32(self.norm2, "weight"), copy, self.eps, self.mult, 1.0)


class DafovikModel(HybridModel):
    config_class = DafovikConfig
    _no_split_modules = ["DafovikLayer"]
    layer_cls = DafovikLayer
    norm_centre = 0.0


class DafovikForCausalLM(HybridForCausalLM):
    config_class = DafovikConfig
    _no_split_modules = ["DafovikLayer"]
    model_cls = DafovikModel


__all__ = ["DafovikConfig", "DafovikForCausalLM", "DafovikModel"]
