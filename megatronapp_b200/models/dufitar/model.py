"""Dufitar: a decoder-only language model over an fp32 residual stream with a squashing norm (``tanh(alpha x) * w + b``, no
statistics) before and after every sublayer and one multiplier on all additions.  Two kinds of mixer, both with a sliding window:
grouped-query attention with YaRN-scaled rotary positions on a part of each head, and latent attention with a rotated key part
shared by the heads, a learned sink in the softmax denominator and an elementwise output gate, whose layers may read the latents of
an earlier one.  Feed-forwards are dense and gated by the tanh form of GELU.  The output layer is the embedding table.

Assembled from the framework's parts: ``LanguageModelEmbedding``, ``SandwichF32Block`` of ``SandwichF32Layer`` with
``WindowAttention`` or ``RotaryLatentAttention`` and ``MLP``, a column-parallel output layer over the embedding's weight.  It follows
the ``GPTModel`` call signature, so the engines, the generation server and the trace replayer drive it like any other language
model.
"""
from __future__ import annotations

from ...parallel.tp_layers import ColumnParallelLinear, RowParallelLinear
from ...transformer.hybrid_layer import SandwichF32Block, SandwichF32Layer
from ...transformer.mla import RotaryLatentAttention
from ...transformer.mlp import MLP, MLPSubmodules
from ...transformer.window_attention import WindowAttention
from ..common.embeddings import LanguageModelEmbedding
from ..common.language_module import LanguageModule
from .config import DufitarConfig

_MLP_SUB = MLPSubmodules(linear_fc1=ColumnParallelLinear, linear_fc2=RowParallelLinear)


def build_mixer(dcfg: DufitarConfig, base, index: int):
    l = dcfg.layers[index]
    mx = l.mixer
    rot, heads, window = mx.get("rot") or {}, int(mx["heads"]), int((mx.get("mask") or {}).get("size") or 0)
    if l.type == "attention":
        return WindowAttention(base, index, heads, int(mx.get("kv_heads", heads)), int(mx["dim"]), int(mx.get("vdim", mx["dim"])),
                               float(mx["scale"]), window, sink=False, slope_exponent=None, qk_norm=False, head_gate=False, bias=False,
                               eps=dcfg.norm_eps, rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
                               rot_scaling=rot.get("scaling"), interleaved=True)
    if l.type == "latent_attention":
        return RotaryLatentAttention(base, index, heads, int(mx["dim"]), int(mx["rot_dim"]), int(mx["vdim"]), int(mx["kv_rank"]), None,
                                     float(mx["scale"]), float(rot.get("base", 10000.0)), rot.get("scaling"), int(mx["rot_dim"]),
                                     interleaved=True, eps=dcfg.norm_eps, window=window, sink=True, element_gate=True,
                                     kv_source_layer=mx.get("kv_from"))
    raise ValueError(f"unknown mixer type {l.type!r}")


def build_mlp(dcfg: DufitarConfig, base, index: int):
    mlp = dcfg.layers[index].mlp
    return MLP(dcfg.mlp_transformer_config(base, mlp), _MLP_SUB) if mlp else None


class DufitarModel(LanguageModule):
    def __init__(self, dcfg: DufitarConfig, config=None, pre_process: bool = True, post_process: bool = True,
                 parallel_output: bool = False, max_sequence_length: int = 0):
        config = config or dcfg.base_transformer_config()
        super().__init__(config)
        self.dcfg = dcfg
        self.vocab_size, self.max_sequence_length = dcfg.vocab, max_sequence_length
        self.pre_process, self.post_process = pre_process, post_process
        self.share_embeddings_and_output_weights = True
        self.model_type = "encoder_or_decoder"
        if pre_process:
            self.embedding = LanguageModelEmbedding(config, dcfg.vocab, max_sequence_length, "none")
        builders = [(lambda i: SandwichF32Layer(config, i, build_mixer(dcfg, config, i), build_mlp(dcfg, config, i), dcfg.residual_mult))
                    for _ in dcfg.layers]
        self.decoder = SandwichF32Block(config, builders, post_process=post_process, input_scale=dcfg.embedding_scale)
        if post_process:
            self.output_layer = ColumnParallelLinear(config.hidden_size, dcfg.vocab, config=config, init_method=config.init_method, bias=False,
                                                     skip_bias_add=False, gather_output=not parallel_output,
                                                     skip_weight_param_allocation=pre_process)
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
        logits, _ = self.output_layer(h, weight=self.shared_embedding_or_output_weight())
        if labels is None:
            return logits.transpose(0, 1).contiguous()
        return self.compute_language_model_loss(labels, logits)
