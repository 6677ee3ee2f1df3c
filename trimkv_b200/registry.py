"""Model classes by the name a ``config.json`` gives: ``architecture``, ``architectures[0]`` or ``model_type``."""
from __future__ import annotations

import json
import os

import torch

from .modeling_dafovik import DafovikForCausalLM
from .modeling_llama import TrimKVLlamaForCausalLM
from .modeling_lonulix import LonulixForCausalLM
from .modeling_phi3 import TrimKVPhi3ForCausalLM
from .modeling_qwen3 import TrimKVQwen3ForCausalLM

MODEL_CLASSES = {
    "Dafovik": DafovikForCausalLM, "dafovik": DafovikForCausalLM, "DafovikForCausalLM": DafovikForCausalLM,
    "Lonulix": LonulixForCausalLM, "lonulix": LonulixForCausalLM, "LonulixForCausalLM": LonulixForCausalLM,
    "TrimKVQwen3ForCausalLM": TrimKVQwen3ForCausalLM, "Qwen3ForCausalLM": TrimKVQwen3ForCausalLM, "qwen3": TrimKVQwen3ForCausalLM,
    "TrimKVLlamaForCausalLM": TrimKVLlamaForCausalLM, "LlamaForCausalLM": TrimKVLlamaForCausalLM, "llama": TrimKVLlamaForCausalLM,
    "TrimKVPhi3ForCausalLM": TrimKVPhi3ForCausalLM, "Phi3ForCausalLM": TrimKVPhi3ForCausalLM, "phi3": TrimKVPhi3ForCausalLM,
}


def model_class(path: str):
    """The class that serves the checkpoint folder ``path``."""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    names = [cfg.get("architecture"), *(cfg.get("architectures") or []), cfg.get("model_type")]
    for name in names:
        if name in MODEL_CLASSES:
            return MODEL_CLASSES[name]
    raise KeyError(f"{path}: no model class for {[n for n in names if n]} (known: {sorted(MODEL_CLASSES)})")


def load_model(path: str, dtype=torch.bfloat16, device="cuda", **kwargs):
    """``from_pretrained`` of the class the folder's ``config.json`` names, on ``device``, ready to generate."""
    return model_class(path).from_pretrained(path, dtype=dtype, **kwargs).to(device).eval()


__all__ = ["MODEL_CLASSES", "load_model", "model_class"]
