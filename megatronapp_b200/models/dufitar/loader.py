"""Weight loading for Dufitar models: the mapping from checkpoint tensor names to the modules' (fused) parameters.

Checkpoint names: ``embed`` (also the output layer), and per layer ``l<i>.mix.<name>``, ``l<i>.mlp.<name>`` and the norms ``l<i>.norm1 /
.norm1b / .norm2 / .norm2b``, like ``final.norm`` each with ``.alpha`` and ``.b`` beside the weight.  Linear weights are stored ``[out, in]``
like the framework's linears, so a mapping is a copy into a (row slice of a) parameter:

* attention: ``q, k, v`` are the row segments of the fused ``in_proj``; ``o``;
* latent attention: ``q, dkv, g`` are the segments of ``in_proj`` (no ``dkv`` in a layer that reads another layer's latents);
  ``dkv.norm, uk, uv, sink, o``;
* feed-forward: ``gate`` and ``up`` are the halves of ``linear_fc1``, ``down`` is ``linear_fc2``.

Sizes that ``config.json`` omits are read from the tensors' shapes.
"""
from __future__ import annotations

import json
import os
from typing import Dict

import torch

from ..zikunex.loader import _copy, read_safetensors


def shapes_into_config(config: dict, shapes: Dict[str, tuple]) -> dict:
    """Fill sizes that only the tensors carry into the config."""
    if "embed" in shapes:
        config.setdefault("vocab", int(shapes["embed"][0]))
        config.setdefault("width", int(shapes["embed"][1]))
    for i, l in enumerate(config["layers"]):
        mx, mlp = l["mixer"], l.get("mlp")
        if l["type"] == "latent_attention" and "kv_rank" not in mx and f"l{i}.mix.uk" in shapes:
            mx["kv_rank"] = int(shapes[f"l{i}.mix.uk"][1])
        if mlp and "ff" not in mlp and f"l{i}.mlp.up" in shapes:
            mlp["ff"] = int(shapes[f"l{i}.mlp.up"][0])
    return config


def load_dufitar_weights(model, tensors: Dict[str, torch.Tensor], strict: bool = True):
    """Copy checkpoint tensors into ``model`` (a ``DufitarModel`` on a single tensor-parallel rank).  A tensor the model
    needs must be there; tensors the model has no parameter for raise under ``strict`` and are returned otherwise."""
    used = set()

    def put(param, name, rows=None):
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        used.add(name)
        _copy(param, tensors[name], name, rows)

    def put_norm(norm, name):
        put(norm.weight, name), put(norm.bias, name + ".b"), put(norm.alpha, name + ".alpha")

    put(model.embedding.word_embeddings.weight, "embed")
    put_norm(model.decoder.final_norm, "final.norm")
    for i, layer in enumerate(model.decoder.layers):
        p, mx = f"l{i}.mix.", layer.mixer
        put_norm(layer.input_norm, f"l{i}.norm1"), put_norm(layer.mixer_norm, f"l{i}.norm1b")
        at = 0
        for seg, n in mx.segments():
            put(mx.in_proj.weight, p + seg, (at, at + n))
            at += n
        if model.dcfg.layers[i].type == "attention":
            put(mx.out_proj.weight, p + "o")
        else:
            if mx.kv_source_layer is None:
                put(mx.kv_norm_weight, p + "dkv.norm")
            put(mx.linear_k_up_proj.weight, p + "uk"), put(mx.linear_v_up_proj.weight, p + "uv")
            put(mx.sink, p + "sink"), put(mx.linear_proj.weight, p + "o")
        if layer.mlp is None:
            continue
        put_norm(layer.pre_mlp_norm, f"l{i}.norm2"), put_norm(layer.mlp_norm, f"l{i}.norm2b")
        m, fc1 = f"l{i}.mlp.", layer.mlp.linear_fc1.weight
        half = fc1.shape[0] // 2
        put(fc1, m + "gate", (0, half)), put(fc1, m + "up", (half, 2 * half)), put(layer.mlp.linear_fc2.weight, m + "down")
    extra = sorted(set(tensors) - used)
    if extra and strict:
        raise ValueError(f"checkpoint tensors without a parameter: {extra[:8]}{' ...' if len(extra) > 8 else ''}")
    return extra


def load_model_dir(path: str, params_dtype=torch.bfloat16, device=None, **config_overrides):
    """Build a ``DufitarModel`` from a folder with ``config.json`` (+ ``model.safetensors``: without it the weights stay
    at their random initialisation) and move it to ``device``."""
    from ...parallel import state as ps
    from .config import DufitarConfig
    from .model import DufitarModel

    if not ps.model_parallel_is_initialized():
        ps.initialize_model_parallel(1, 1)
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    st = os.path.join(path, "model.safetensors")
    tensors = read_safetensors(st) if os.path.exists(st) else None
    raw = shapes_into_config(raw, {k: tuple(v.shape) for k, v in tensors.items()} if tensors is not None else {})
    dcfg = DufitarConfig.from_dict(raw)
    base = dcfg.base_transformer_config(params_dtype, use_cpu_initialization=True, perform_initialization=tensors is None,
                                        **config_overrides)
    model = DufitarModel(dcfg, base)
    if tensors is not None:
        extra = load_dufitar_weights(model, tensors, strict=False)
        if extra:
            import sys

            print(f"[dufitar] {len(extra)} checkpoint tensors have no parameter and were ignored: {extra[:4]}", file=sys.stderr)
    if device is not None:
        model = model.to(device)
    return model.eval()
