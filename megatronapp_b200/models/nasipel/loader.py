"""Weight loading for Nasipel models: the mapping from checkpoint tensor names to the modules' (fused) parameters.

Checkpoint names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.norm1 / .norm2``, ``l<i>.rg1 / .rg1.b / .rg2 / .rg2.b``,
``l<i>.mix.<name>``, ``l<i>.mlp.<name>``.  Linear weights are stored ``[out, in]`` like the framework's linears, so a mapping is
a copy into a (row slice of a) parameter:

* attention: ``q, k, v`` are the row segments of the fused ``in_proj``; ``pb`` the bias per head; ``o``;
* rglru: ``y, x`` (and ``y.b, x.b``) are the segments of ``in_proj``; ``conv, conv.b, lam, o``; ``ra, ri`` (and ``ra.b, ri.b``) the two
  matrices of every gate block;
* latent attention: ``dq, dkv, g`` are the segments of ``in_proj``; ``dq.norm, dkv.norm, uq, uk, uv, o``;
* feed-forward: ``router, correction``; ``e<j>.gate`` and ``e<j>.up`` are the halves of expert ``j``'s rows of the grouped
  ``weight1``, ``e<j>.down`` its rows of ``weight2``.

Sizes that ``config.json`` omits (latent ranks, convolution taps, gate blocks) are read from the tensors' shapes.
"""
from __future__ import annotations

import json
import os
from typing import Dict

import torch

from ..zikunex.loader import _copy, read_safetensors


def shapes_into_config(config: dict, shapes: Dict[str, tuple]) -> dict:
    """Fill sizes that only the tensors carry into the mixer dicts."""
    for i, l in enumerate(config["layers"]):
        mx = l["mixer"]
        for kind, key, name, axis in (("latent_attention", "q_rank", "dq", 0), ("latent_attention", "kv_rank", "uk", 1),
                                      ("rglru", "conv", "conv", 1), ("rglru", "width", "lam", 0), ("rglru", "blocks", "ra", 0)):
            t = shapes.get(f"l{i}.mix.{name}")
            if l["type"] == kind and key not in mx and t is not None:
                mx[key] = int(t[axis])
    return config


def load_nasipel_weights(model, tensors: Dict[str, torch.Tensor], strict: bool = True):
    """Copy checkpoint tensors into ``model`` (a ``NasipelModel`` on a single tensor-parallel rank).  A tensor the model
    needs must be there; tensors the model has no parameter for raise under ``strict`` and are returned otherwise."""
    used = set()

    def put(param, name, rows=None):
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        used.add(name)
        _copy(param, tensors[name], name, rows)

    def segments(param, pre, segs, suffix=""):
        o = 0
        for seg, n in segs:
            put(param, f"{pre}{seg}{suffix}", (o, o + n))
            o += n

    put(model.embedding.word_embeddings.weight, "embed")
    put(model.output_layer.weight, "head")
    put(model.decoder.final_norm_weight, "final.norm")
    for i, layer in enumerate(model.decoder.layers):
        put(layer.input_norm_weight, f"l{i}.norm1")
        put(layer.mixer_gate.weight, f"l{i}.rg1"), put(layer.mixer_gate.bias, f"l{i}.rg1.b")
        p, mx, kind = f"l{i}.mix.", layer.mixer, model.ncfg.layers[i].type
        segments(mx.in_proj.weight, p, mx.segments())
        if kind == "attention":
            named = (("pb", mx.head_bias), ("o", mx.out_proj.weight))
        elif kind == "rglru":
            segments(mx.in_proj.bias, p, mx.segments(), ".b")
            named = (("conv", mx.conv_weight), ("conv.b", mx.conv_bias), ("ra", mx.gate_weight[:, 0]), ("ri", mx.gate_weight[:, 1]),
                     ("ra.b", mx.gate_bias[:, 0]), ("ri.b", mx.gate_bias[:, 1]), ("lam", mx.lam), ("o", mx.out_proj.weight))
        else:
            named = (("dq.norm", mx.q_norm_weight), ("dkv.norm", mx.kv_norm_weight), ("uq", mx.linear_q_up_proj.weight),
                     ("uk", mx.linear_k_up_proj.weight), ("uv", mx.linear_v_up_proj.weight), ("o", mx.linear_proj.weight))
        for n, prm in named:
            put(prm, p + n)
        if layer.mlp is None:
            continue
        put(layer.pre_mlp_norm_weight, f"l{i}.norm2")
        put(layer.mlp_gate.weight, f"l{i}.rg2"), put(layer.mlp_gate.bias, f"l{i}.rg2.b")
        m, router, ex, h = f"l{i}.mlp.", layer.mlp.router, layer.mlp.experts, model.config.hidden_size
        put(router.weight, m + "router"), put(router.expert_bias, m + "correction")
        for e in range(ex.num_local_experts):
            put(ex.weight1, f"{m}e{e}.gate", (e * ex.fc1_out, e * ex.fc1_out + ex.ffn))
            put(ex.weight1, f"{m}e{e}.up", (e * ex.fc1_out + ex.ffn, (e + 1) * ex.fc1_out))
            put(ex.weight2, f"{m}e{e}.down", (e * h, (e + 1) * h))
    extra = sorted(set(tensors) - used)
    if extra and strict:
        raise ValueError(f"checkpoint tensors without a parameter: {extra[:8]}{' ...' if len(extra) > 8 else ''}")
    return extra


def load_model_dir(path: str, params_dtype=torch.bfloat16, device=None, **config_overrides):
    """Build a ``NasipelModel`` from a folder with ``config.json`` (+ ``model.safetensors``: without it the weights stay
    at their random initialisation) and move it to ``device``."""
    from ...parallel import state as ps
    from .config import NasipelConfig
    from .model import NasipelModel

    if not ps.model_parallel_is_initialized():
        ps.initialize_model_parallel(1, 1)
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    st = os.path.join(path, "model.safetensors")
    tensors = read_safetensors(st) if os.path.exists(st) else None
    raw = shapes_into_config(raw, {k: tuple(v.shape) for k, v in tensors.items()} if tensors is not None else {})
    ncfg = NasipelConfig.from_dict(raw)
    base = ncfg.base_transformer_config(params_dtype, use_cpu_initialization=True, perform_initialization=tensors is None,
                                        **config_overrides)
    model = NasipelModel(ncfg, base)
    if tensors is not None:
        extra = load_nasipel_weights(model, tensors, strict=False)
        if extra:
            import sys

            print(f"[nasipel] {len(extra)} checkpoint tensors have no parameter and were ignored: {extra[:4]}", file=sys.stderr)
    if device is not None:
        model = model.to(device)
    return model.eval()
