"""What the hybrid decoders share: models whose layers are of several kinds, each with its own state, over a residual stream
that is fp32 whatever the model type (the products read its copy in the model type).

A design supplies a configuration (``HybridConfig``: order of layers, sizes and constants, all from ``config.json``), a layer
(``forward(stream, copy, batch, data)``, ``checkpoint()``, ``mix.state()``) and a final norm; this module does the rest: loading
and saving, the packed step over ``HybridStateCache`` that serves prompts, portions of prompts and decoding, the HF call form,
and the one-token step of ``generate``, ``generate_greedy`` and ``GreedyDecoder``.  bf16 models run the tensor-core kernels, fp32
models the fp32 forms of the same kernels.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional, Sequence

import torch
import torch.nn.functional as F
from torch import nn
from transformers import PretrainedConfig
from transformers.modeling_outputs import BaseModelOutputWithPast, CausalLMOutputWithPast

from . import ops
from .mixers import FusedProjection, Mixer, as_f32
from .modeling_trimkv import TrimKVForCausalLM, TrimKVPreTrainedModel
from .state_cache import HybridStateCache, StepBatch


class HybridConfig(PretrainedConfig):
    """``layers``: one entry per layer with ``type`` (a key of ``mixers``), ``mixer`` (its sizes and constants) and ``mlp`` (a
    mapping whose ``kind`` is one of ``feed_forwards``, or None); ``norm.eps``, ``vocab``, ``width``.  ``checkpoint_keys`` are the
    entries a ``config.json`` holds."""

    architecture = ""
    mixers = {}
    feed_forwards = {}
    checkpoint_keys = ("layers", "norm", "vocab", "width")

    def __init__(self, layers: Optional[List[dict]] = None, norm: Optional[dict] = None, vocab: int = 256, width: int = 64, **kwargs):
        self.layers = list(layers or [])
        self.norm = dict(norm or {"eps": 1e-6})
        self.vocab, self.width = int(vocab), int(width)
        for i, layer in enumerate(self.layers):
            if layer["type"] not in self.mixers:
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r} (known: {sorted(self.mixers)})")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") not in self.feed_forwards:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r} (known: {sorted(self.feed_forwards)} or null)")
        # the names the rest of the framework and HF generation read
        self.vocab_size, self.hidden_size, self.num_hidden_layers = self.vocab, self.width, len(self.layers)
        self.initializer_range = kwargs.pop("initializer_range", 0.02)
        self.fused_decode_step = kwargs.pop("fused_decode_step", False)
        self.compress_memory = False                     # nothing of these designs' state is ever evicted
        kwargs.pop("architecture", None)
        kwargs.setdefault("tie_word_embeddings", False)
        super().__init__(**kwargs)

    @classmethod
    def from_pretrained(cls, path, **kwargs):
        file = os.path.join(path, "config.json") if os.path.isdir(path) else path
        with open(file) as f:
            return cls(**{**json.load(f), **kwargs})

    def checkpoint_dict(self) -> dict:
        return {"architecture": self.architecture, **{k: getattr(self, k) for k in self.checkpoint_keys}}


class StreamNorm(nn.Module):
    """Weight of an RMS norm of the stream, stored around ``centre`` (the kernels add ``1 - centre``)."""

    def __init__(self, width: int, centre: float = 1.0):
        super().__init__()
        self.centre = centre
        self.weight = nn.Parameter(torch.full((width,), float(centre)))


class HybridPreTrainedModel(TrimKVPreTrainedModel):
    config_class = HybridConfig

    def _init_weights(self, module):
        if isinstance(module, StreamNorm):
            nn.init.constant_(module.weight, module.centre)
        elif hasattr(module, "checkpoint") and hasattr(module, "reset_parameters"):       # mixers, feed-forwards, layers
            module.reset_parameters(self.config.initializer_range)
        elif not isinstance(module, FusedProjection):     # its owner fills it
            super()._init_weights(module)

    @classmethod
    def from_pretrained(cls, pretrained_model_name_or_path, *, dtype=None, torch_dtype=None, device=None, device_map=None, **kwargs):
        """``config.json`` and ``model.safetensors`` of a local folder.  Every tensor the configuration calls for must be there
        in the right shape, and nothing else."""
        path = pretrained_model_name_or_path
        if not os.path.isdir(path):
            raise ValueError(f"Path {path} does not exist.")
        config = cls.config_class.from_pretrained(path, **kwargs)
        dtype = dtype or torch_dtype or torch.bfloat16
        if isinstance(dtype, str):
            dtype = getattr(torch, dtype)
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: this design runs in bfloat16 or float32")
        device = torch.device(device if device is not None else (device_map if isinstance(device_map, (str, torch.device)) else "cpu"))
        with torch.device("meta"):
            model = cls(config)
        model = model.to(dtype).to_empty(device=device)
        model.load_checkpoint(os.path.join(path, "model.safetensors"))
        return model.eval()


class HybridModel(HybridPreTrainedModel):
    layer_cls = None
    embed_scale, norm_groups, norm_centre = 1.0, 1, 1.0

    def __init__(self, config: HybridConfig):
        super().__init__(config)
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.layers = nn.ModuleList([self.layer_cls(config, i) for i in range(len(config.layers))])
        self.norm = StreamNorm(config.width, self.norm_centre)
        self.post_init()

    def get_input_embeddings(self):
        return self.embed_tokens

    def set_input_embeddings(self, value):
        self.embed_tokens = value

    def step(self, ids: torch.Tensor, batch: StepBatch, cache: HybridStateCache, layers_out: Optional[list] = None) -> torch.Tensor:
        """Packed token ids ``[tokens]`` of a begun step -> the fp32 residual stream ``[tokens, width]``."""
        w = self.embed_tokens.weight
        stream = torch.empty(batch.tokens, w.shape[1], dtype=torch.float32, device=w.device)
        copy = None if w.dtype == torch.float32 else torch.empty(batch.tokens, w.shape[1], dtype=w.dtype, device=w.device)
        ops.embed_stream(ids, w, stream, copy, batch.status, self.embed_scale)
        for i, layer in enumerate(self.layers):
            layer(stream, copy, batch, cache.arrays(i))
            if layers_out is not None:
                layers_out.append(stream.clone())
        return stream

    def final_norm(self, stream: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The normed stream in the model type, of all rows or of those named by ``rows`` (int32)."""
        w = self.embed_tokens.weight
        out = torch.empty(stream.shape[0] if rows is None else rows.shape[0], w.shape[1], dtype=w.dtype, device=w.device)
        ops.stream_norm(stream, rows, as_f32(self.norm, "weight"), out, self.config.norm["eps"], 1.0 - self.norm_centre, self.norm_groups)
        return out

    def compress_after_forward(self, past_key_values) -> None:
        """Windows and states are bounded by construction: nothing to evict at the end of a step."""

    def forward(self, input_ids=None, attention_mask=None, past_key_values: Optional[HybridStateCache] = None, **_unused):
        return BaseModelOutputWithPast(last_hidden_state=None, past_key_values=past_key_values)


class HybridForCausalLM(HybridPreTrainedModel, TrimKVForCausalLM):
    model_cls = HybridModel
    cache_cls = HybridStateCache
    decode_dtypes = (torch.bfloat16, torch.float32)
    _tied_weights_keys = {}

    # ------------------------------------------------------------------ checkpoints
    def checkpoint_tensors(self) -> Dict[str, torch.Tensor]:
        """The names a checkpoint uses -> the parameters (or the parts of fused ones) they fill."""
        m = self.model
        out = {"embed": m.embed_tokens.weight, "final.norm": m.norm.weight, "head": self.lm_head.weight}
        for i, layer in enumerate(m.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.checkpoint().items()})
        return out

    @torch.no_grad()
    def load_checkpoint(self, file: str) -> None:
        from safetensors import safe_open
        want = self.checkpoint_tensors()
        for p in self.parameters():                       # the padding rows of fused projections are not in a checkpoint
            p.zero_()
        with safe_open(file, framework="pt") as f:
            have = set(f.keys())
            if have != set(want):
                raise ValueError(f"{file}: missing tensors {sorted(set(want) - have)}, unexpected tensors {sorted(have - set(want))}")
            for name, param in want.items():
                t = f.get_tensor(name)
                if t.shape != param.shape:
                    raise ValueError(f"{file}: {name} has shape {tuple(t.shape)}, the configuration says {tuple(param.shape)}")
                param.copy_(t)

    def save_checkpoint(self, path: str) -> None:
        """``config.json`` and ``model.safetensors`` (bfloat16) as ``from_pretrained`` reads them."""
        from safetensors.torch import save_file
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.config.checkpoint_dict(), f, indent=1)
        save_file({k: v.detach().to(torch.bfloat16).cpu().contiguous().clone() for k, v in self.checkpoint_tensors().items()},
                  os.path.join(path, "model.safetensors"))

    # ------------------------------------------------------------------ steps
    def new_cache(self, device=None, capacity_tokens: int = 0) -> HybridStateCache:
        return HybridStateCache([layer.mix.state() for layer in self.model.layers], device or self.device,
                                self.lm_head.weight.dtype, capacity_tokens)

    def head(self, normed: torch.Tensor) -> torch.Tensor:
        """Logits in fp32."""
        w = self.lm_head.weight
        return F.linear(normed, w) if w.dtype == torch.float32 else torch.mm(normed, w.t(), out_dtype=torch.float32)

    @torch.no_grad()
    def forward_packed(self, ids: torch.Tensor, cache: HybridStateCache, lengths: Optional[Sequence[int]],
                       rows: Optional[Sequence[int]] = None, want: Optional[Sequence[int]] = None,
                       layers_out: Optional[list] = None) -> torch.Tensor:
        """One step of any requests of the batch: packed ids ``[sum(lengths)]`` -> fp32 logits ``[wanted, vocab]``.
        ``lengths`` None: one token per request.  ``want``: packed places (None: every token)."""
        if not ids.is_cuda:
            raise ops._lib.TrimKVNativeError("this model runs on CUDA tensors only (no CPU path)")
        batch = cache.begin(lengths, rows)
        if ids.shape[0] != batch.tokens:
            raise ValueError(f"{ids.shape[0]} token ids for {batch.tokens} tokens")
        stream = self.model.step(ids, batch, cache, layers_out)
        at = None
        if want is not None:
            if len(want) == 0:
                return stream.new_empty(0, self.config.vocab)
            at = torch.tensor(list(want), dtype=torch.int32).to(ids.device, non_blocking=True)
        return self.head(self.model.final_norm(stream, at))

    def decode_step(self, ids: torch.Tensor, cache: HybridStateCache) -> torch.Tensor:
        """One token of every request of the batch, ids ``[B]`` on the device -> fp32 logits ``[B, vocab]``.  Recordable in a
        CUDA graph once it has run on this batch."""
        stream = self.model.step(ids, cache.begin(None), cache)
        return self.head(self.model.final_norm(stream))

    def forward(self, input_ids=None, attention_mask=None, position_ids=None, past_key_values=None, inputs_embeds=None,
                use_cache=None, cache_position=None, logits_to_keep=0, **kwargs):
        """HF call form.  ``attention_mask`` ``[B, >= S]`` marks the padding of unequal prompts, on either side; positions are
        counted per request.  ``logits_to_keep=1``: every request's last token; 0: all places (zeros at padding)."""
        if input_ids is None or inputs_embeds is not None:
            raise ValueError("this model takes input_ids")
        cache = past_key_values if past_key_values is not None else self.new_cache(input_ids.device)
        bsz, width = input_ids.shape
        if cache._batch == 0:
            cache.open(bsz)
        if cache._batch != bsz:
            raise ValueError(f"{bsz} rows for a cache of {cache._batch} requests")
        step = self._fused_step_for(input_ids, cache, inputs_embeds, kwargs)
        if step is not None:
            logits = step(cache, input_ids, torch.zeros(1, dtype=torch.int64, device=input_ids.device))
            return CausalLMOutputWithPast(logits=logits[:, None, :], past_key_values=cache)
        if width == 1:
            logits = self.forward_packed(input_ids.reshape(-1), cache, None)
            return CausalLMOutputWithPast(logits=logits[:, None, :], past_key_values=cache)
        live = None
        if attention_mask is not None and attention_mask.dim() == 2:
            live = attention_mask[:, -width:].bool()
            if bool(live.all()):
                live = None
        lengths = [width] * bsz if live is None else live.sum(1).tolist()
        rows = [b for b in range(bsz) if lengths[b] > 0]  # a portion that is padding only for some requests
        ids = input_ids.reshape(-1) if live is None else input_ids[live]
        counts = [lengths[b] for b in rows]
        if logits_to_keep == 1:
            ends, at = [], -1
            for n in counts:
                at += n
                ends.append(at)
            got = self.forward_packed(ids, cache, counts, rows, ends)
            logits = got if len(rows) == bsz else got.new_zeros(bsz, got.shape[1]).index_copy_(0, torch.tensor(rows, device=got.device), got)
            return CausalLMOutputWithPast(logits=logits[:, None, :], past_key_values=cache)
        got = self.forward_packed(ids, cache, counts, rows)
        if live is None:
            logits = got.view(bsz, width, -1)
        else:
            logits = got.new_zeros(bsz, width, got.shape[1])
            logits[live] = got
        if not isinstance(logits_to_keep, int):
            logits = logits[:, logits_to_keep]
        elif logits_to_keep:
            logits = logits[:, -logits_to_keep:]
        return CausalLMOutputWithPast(logits=logits, past_key_values=cache)

    def _decode_step_cls(self):
        from .decoder import HybridDecodeStep
        return HybridDecodeStep


__all__ = ["HybridConfig", "HybridForCausalLM", "HybridModel", "HybridPreTrainedModel", "StreamNorm"]
