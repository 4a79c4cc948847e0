"""Configuration of Dufitar models: the ``config.json`` reader and its mapping onto the framework's configs.

``config.json`` keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult`` and ``layers``: a list
whose entries carry ``type`` (``attention`` or ``latent_attention``), the mixer's sizes under ``mixer`` and the feed-forward under ``mlp``
(``null``: none).

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the window), ``rot.dims`` / ``rot.base`` /
  ``rot.scaling`` (``factor``, ``original``, ``fast``, ``slow``; absent: plain rotation).
* ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``mask.size``, ``rot.base``, ``kv_from`` (the layer
  whose latents it reads; absent: its own).
* ``mlp.kind`` ``dense``: ``ff``.
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import torch

from ...config.transformer_config import TransformerConfig
from ...transformer.mlp import gelu_glu

MIXER_TYPES = ("attention", "latent_attention")


@dataclass
class DufitarLayerConfig:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]] = None


@dataclass
class DufitarConfig:
    vocab: int
    width: int
    layers: List[DufitarLayerConfig]
    norm_eps: float = 1e-6
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    architecture: str = "Dufitar"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "DufitarConfig":
        layers: List[DufitarLayerConfig] = []
        for i, l in enumerate(d["layers"]):
            if l["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            if l.get("mlp") and l["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown mlp kind {l['mlp'].get('kind')!r}")
            mixer = dict(l["mixer"])
            src = mixer.get("kv_from")
            if src is not None and not (0 <= src < i and layers[src].type == "latent_attention" and layers[src].mixer.get("kv_from") is None):
                raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with latents of its own")
            layers.append(DufitarLayerConfig(l["type"], mixer, dict(l["mlp"]) if l.get("mlp") else None))
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=layers, norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), residual_mult=float(d.get("residual_mult", 1.0)),
                   architecture=d.get("architecture", "Dufitar"))

    @classmethod
    def from_json(cls, path: str) -> "DufitarConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f))

    # -- mapping onto the framework's TransformerConfig ---------------------------------------------------------------------
    def base_transformer_config(self, params_dtype=torch.bfloat16, use_cpu_initialization: Optional[bool] = None,
                                perform_initialization: bool = True, **overrides) -> TransformerConfig:
        cpu = (not torch.cuda.is_available()) if use_cpu_initialization is None else use_cpu_initialization
        kw = dict(num_layers=len(self.layers), hidden_size=self.width, num_attention_heads=1, kv_channels=self.width,
                  ffn_hidden_size=self.width, normalization="RMSNorm", layernorm_epsilon=self.norm_eps, add_bias_linear=False,
                  gated_linear_unit=True, activation_func=gelu_glu, hidden_dropout=0.0, attention_dropout=0.0,
                  params_dtype=params_dtype, bf16=params_dtype == torch.bfloat16, fp16=params_dtype == torch.float16,
                  fp32_residual_connection=True, use_cpu_initialization=cpu, perform_initialization=perform_initialization,
                  bias_activation_fusion=False)
        kw.update(overrides)
        return TransformerConfig(**kw)

    @staticmethod
    def mlp_transformer_config(base: TransformerConfig, mlp: Dict[str, Any]) -> TransformerConfig:
        return dataclasses.replace(base, ffn_hidden_size=int(mlp["ff"]), num_moe_experts=None)
