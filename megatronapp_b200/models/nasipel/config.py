"""Configuration of Nasipel models: the ``config.json`` reader and its mapping onto the framework's configs.

``config.json`` keys: ``architecture``, ``vocab``, ``width``, ``norm.eps`` and ``layers``: a list whose entries carry ``type``
(``attention``, ``rglru`` or ``latent_attention``), the mixer's sizes under ``mixer`` and the feed-forward under ``mlp``
(``null``: none).

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap`` (absent: no cap), ``rot.dims`` / ``rot.base``.
* ``rglru``: ``width``, ``blocks`` (parts of the block-diagonal gates), ``conv`` (taps).
* ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot.base``, ``rot.scaling``
  (``factor``, ``original``, ``fast``, ``slow``; absent: plain rotation).
* ``mlp.kind`` ``moe``: ``expert.ff``, ``router.experts``, ``router.top``, ``router.scale``, ``router.groups.count`` / ``keep``.
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import torch
import torch.nn.functional as F

from ...config.transformer_config import TransformerConfig

MIXER_TYPES = ("attention", "rglru", "latent_attention")
DECAY_SCALE = 8.0               # log a = -DECAY_SCALE * r * softplus(lam) in the recurrent unit


@dataclass
class NasipelLayerConfig:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]] = None


@dataclass
class NasipelConfig:
    vocab: int
    width: int
    layers: List[NasipelLayerConfig]
    norm_eps: float = 1e-5
    architecture: str = "Nasipel"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NasipelConfig":
        layers = []
        for i, l in enumerate(d["layers"]):
            if l["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            if l.get("mlp") and l["mlp"].get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown mlp kind {l['mlp'].get('kind')!r}")
            layers.append(NasipelLayerConfig(l["type"], dict(l["mixer"]), dict(l["mlp"]) if l.get("mlp") else None))
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), layers=layers,
                   norm_eps=float((d.get("norm") or {}).get("eps", 1e-5)), architecture=d.get("architecture", "Nasipel"))

    @classmethod
    def from_json(cls, path: str) -> "NasipelConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f))

    # -- mapping onto the framework's TransformerConfig ---------------------------------------------------------------------
    def base_transformer_config(self, params_dtype=torch.bfloat16, use_cpu_initialization: Optional[bool] = None,
                                perform_initialization: bool = True, **overrides) -> TransformerConfig:
        cpu = (not torch.cuda.is_available()) if use_cpu_initialization is None else use_cpu_initialization
        kw = dict(num_layers=len(self.layers), hidden_size=self.width, num_attention_heads=1, kv_channels=self.width,
                  ffn_hidden_size=self.width, normalization="LayerNorm", layernorm_epsilon=self.norm_eps, add_bias_linear=False,
                  gated_linear_unit=True, activation_func=F.silu, hidden_dropout=0.0, attention_dropout=0.0,
                  params_dtype=params_dtype, bf16=params_dtype == torch.bfloat16, fp16=params_dtype == torch.float16,
                  fp32_residual_connection=True, use_cpu_initialization=cpu, perform_initialization=perform_initialization,
                  bias_activation_fusion=False)
        kw.update(overrides)
        return TransformerConfig(**kw)

    @staticmethod
    def mlp_transformer_config(base: TransformerConfig, mlp: Dict[str, Any]) -> TransformerConfig:
        """Mixture of SiLU-gated experts: logistic scores in fp32, the choice by score + correction (the router's expert bias)
        within the best groups (ranked by their two best choice scores), weights renormalised and scaled."""
        r, ex = mlp["router"], mlp["expert"]
        groups = r.get("groups") or {}
        return dataclasses.replace(
            base, num_moe_experts=int(r["experts"]), moe_router_topk=int(r["top"]), moe_ffn_hidden_size=int(ex["ff"]),
            ffn_hidden_size=int(ex["ff"]), gated_linear_unit=True, activation_func=F.silu, moe_router_pre_softmax=False,
            moe_router_score_function="sigmoid", moe_router_dtype="fp32", moe_router_enable_expert_bias=True,
            moe_router_num_groups=int(groups["count"]) if groups else None, moe_router_group_topk=int(groups["keep"]) if groups else None,
            moe_router_group_score="top2_sum", moe_router_renormalize=True, moe_router_topk_scaling_factor=float(r.get("scale", 1.0)),
            moe_router_load_balancing_type="none", moe_aux_loss_coeff=0.0, moe_token_dispatcher_type="fused", moe_grouped_gemm=True)
