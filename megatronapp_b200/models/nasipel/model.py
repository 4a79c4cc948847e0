"""Nasipel: a decoder-only hybrid over an fp32 residual stream.  In every layer mixer and feed-forward stand side by side, each
behind a layer norm of its own (same input, no bias), each result gated element by element by a logistic function of a
projection of that sublayer's normed input.  Three kinds of mixer: attention with logistic weights, rotary queries, keys and
values and a bias per head; Griffin's recurrent block with a real-gated linear recurrent unit and block-diagonal gates;
latent attention with a YaRN-scaled rotated key part shared by the heads and an output gate per head.  Feed-forwards are
mixtures of SiLU-gated experts, chosen by corrected logistic scores inside the best groups.

Assembled from the framework's parts: ``LanguageModelEmbedding``, ``DualNormF32Block`` of ``DualNormF32Layer`` with
``SigmoidAttention``, ``RGLRUMixer`` or ``RotaryLatentAttention``, ``MoELayer`` (``TopKRouter``, fused dispatcher,
``GroupedMLP``), a column-parallel output layer.  It follows the ``GPTModel`` call signature, so the engines, the generation
server and the trace replayer drive it like any other language model.
"""
from __future__ import annotations

from ...moe.experts import GroupedMLP
from ...moe.moe_layer import MoELayer, MoESubmodules
from ...parallel.tp_layers import ColumnParallelLinear, RowParallelLinear
from ...ssm.rglru import RGLRUMixer
from ...transformer.hybrid_layer import DualNormF32Block, DualNormF32Layer
from ...transformer.mla import RotaryLatentAttention
from ...transformer.mlp import MLPSubmodules
from ...transformer.sigmoid_attention import SigmoidAttention
from ...transformer.spec_utils import ModuleSpec
from ..common.embeddings import LanguageModelEmbedding
from ..common.language_module import LanguageModule
from .config import DECAY_SCALE, NasipelConfig

_MLP_SUB = MLPSubmodules(linear_fc1=ColumnParallelLinear, linear_fc2=RowParallelLinear)


def build_mixer(ncfg: NasipelConfig, base, index: int):
    l = ncfg.layers[index]
    mx = l.mixer
    rot = mx.get("rot") or {}
    if l.type == "attention":
        heads = int(mx["heads"])
        return SigmoidAttention(base, index, heads, int(mx.get("kv_heads", heads)), int(mx["dim"]), int(mx.get("vdim", mx["dim"])),
                                float(mx["scale"]), float(mx.get("softcap") or 0.0), int(rot.get("dims", 0)), float(rot.get("base", 10000.0)),
                                rot.get("scaling"), interleaved=False, rotate_values=bool(rot), qk_norm=True, eps=ncfg.norm_eps)
    if l.type == "rglru":
        return RGLRUMixer(base, index, int(mx["width"]), int(mx["blocks"]), int(mx["conv"]), DECAY_SCALE)
    if l.type == "latent_attention":
        return RotaryLatentAttention(base, index, int(mx["heads"]), int(mx["dim"]), int(mx["rot_dim"]), int(mx["vdim"]), int(mx["kv_rank"]),
                                     int(mx["q_rank"]), float(mx["scale"]), float(rot.get("base", 10000.0)), rot.get("scaling"),
                                     int(rot.get("dims", mx["rot_dim"])), interleaved=True, head_gate=True, eps=ncfg.norm_eps)
    raise ValueError(f"unknown mixer type {l.type!r}")


def build_mlp(ncfg: NasipelConfig, base, index: int):
    mlp = ncfg.layers[index].mlp
    if not mlp:
        return None
    return MoELayer(ncfg.mlp_transformer_config(base, mlp), MoESubmodules(experts=ModuleSpec(module=GroupedMLP, submodules=_MLP_SUB)),
                    layer_number=index)


class NasipelModel(LanguageModule):
    def __init__(self, ncfg: NasipelConfig, config=None, pre_process: bool = True, post_process: bool = True,
                 parallel_output: bool = False, max_sequence_length: int = 0):
        config = config or ncfg.base_transformer_config()
        super().__init__(config)
        self.ncfg = ncfg
        self.vocab_size, self.max_sequence_length = ncfg.vocab, max_sequence_length
        self.pre_process, self.post_process = pre_process, post_process
        self.share_embeddings_and_output_weights = False
        self.model_type = "encoder_or_decoder"
        if pre_process:
            self.embedding = LanguageModelEmbedding(config, ncfg.vocab, max_sequence_length, "none")
        builders = [(lambda i: DualNormF32Layer(config, i, build_mixer(ncfg, config, i), build_mlp(ncfg, config, i)))
                    for _ in ncfg.layers]
        self.decoder = DualNormF32Block(config, builders, post_process=post_process)
        if post_process:
            self.output_layer = ColumnParallelLinear(config.hidden_size, ncfg.vocab, config=config, init_method=config.init_method,
                                                     bias=False, skip_bias_add=False, gather_output=not parallel_output)
        self.setup_embeddings_and_output_layer()

    def set_input_tensor(self, t):
        self.decoder.set_input_tensor(t[0] if isinstance(t, (list, tuple)) else t)

    def forward(self, input_ids, position_ids=None, attention_mask=None, decoder_input=None, labels=None,
                inference_context=None, inference_params=None, **_):
        inference_context = inference_context or inference_params
        x = decoder_input
        if x is None and self.pre_process:
            x = self.embedding(input_ids=input_ids, position_ids=position_ids)
        h = self.decoder(x, inference_context=inference_context)
        if not self.post_process:
            return h
        logits, _ = self.output_layer(h)
        if labels is None:
            return logits.transpose(0, 1).contiguous()
        return self.compute_language_model_loss(labels, logits)
