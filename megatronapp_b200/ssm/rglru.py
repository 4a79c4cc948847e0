"""Recurrent block around a real-gated linear recurrent unit (RG-LRU) with block-diagonal gates.

    y = gelu_tanh(W_y h + b_y);   u = conv(W_x h + b_x)             (causal, depth-wise over time, with a bias, no activation)
    r, i = sigmoid(blockdiag(W_r) u + b_r), sigmoid(blockdiag(W_i) u + b_i)
    a = exp(-decay_scale * r * softplus(lam));   S <- a S + sqrt(1 - a^2) i u   (S = 0 before the first token)
    out = W_o (S * y)

De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models".  One fused input
projection with the row segments ``[y | x]``; the state (one fp32 value per channel and sequence, and the convolution's last
``taps - 1`` inputs) lives in the inference context; the gates' sums, decays and the recurrence are fp32.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ..ops import seqmix
from ..parallel.tp_layers import ColumnParallelLinear, RowParallelLinear
from ..transformer.module import MegatronModule
from .gated_delta import packed_tokens, unpacked_tokens


class RGLRUMixer(MegatronModule):
    def __init__(self, config, layer_number: int, width: int, blocks: int, conv_taps: int, decay_scale: float = 8.0):
        super().__init__(config)
        if width % blocks:
            raise ValueError("rg-lru: the width must be a multiple of the number of gate blocks")
        self.layer_number, self.width, self.blocks, self.taps = layer_number, int(width), int(blocks), int(conv_taps)
        self.decay_scale = float(decay_scale)
        self.in_proj = ColumnParallelLinear(config.hidden_size, 2 * self.width, config=config, init_method=config.init_method,
                                            bias=True, skip_bias_add=False, gather_output=False)
        dev, dt_ = self.in_proj.weight.device, config.params_dtype
        n = self.width // self.blocks
        self.conv_weight = nn.Parameter(torch.randn(self.width, self.taps, device=dev).mul_(self.taps ** -0.5).to(dt_))
        self.conv_bias = nn.Parameter(torch.zeros(self.width, device=dev, dtype=dt_))
        # per block: the recurrence gate's matrix and the input gate's, [out, in] each
        self.gate_weight = nn.Parameter(torch.randn(self.blocks, 2, n, n, device=dev).mul_(n ** -0.5).to(dt_))
        self.gate_bias = nn.Parameter(torch.zeros(self.blocks, 2, n, device=dev, dtype=dt_))
        self.lam = nn.Parameter(torch.full((self.width,), -4.0, device=dev).to(dt_))
        self.out_proj = RowParallelLinear(self.width, config.hidden_size, config=config, init_method=config.output_layer_init_method,
                                          bias=False, input_is_parallel=True, skip_bias_add=True)
        self.lam._no_weight_decay = True

    def segments(self):
        """Row counts of the ``[y | x]`` segments of ``in_proj``."""
        return [("y", self.width), ("x", self.width)]

    def forward(self, hidden_states, inference_context=None, cache_index=None, **_):
        s, b = hidden_states.shape[0], hidden_states.shape[1]
        key = self.layer_number if cache_index is None else cache_index
        proj, _ = self.in_proj(hidden_states)
        proj = packed_tokens(proj)
        y_pre, x = proj[:, :self.width], proj[:, self.width:]
        if inference_context is not None:
            if inference_context.is_static_batching():
                raise NotImplementedError("recurrent mixers serve through the dynamic engine")
            pb = inference_context.packed
            window = inference_context.recurrent_state(("rglru.conv", key), (self.taps - 1, self.width), proj.dtype)
            state = inference_context.recurrent_state(("rglru.S", key), (self.width,), torch.float32)
        else:
            pb = seqmix.PackedBatch.dense(s, b, proj.device)
            window = proj.new_zeros(b, self.taps - 1, self.width)
            state = torch.zeros(b, self.width, dtype=torch.float32, device=proj.device)
        u = seqmix.causal_conv(x, self.conv_weight, pb, window, bias=self.conv_bias)
        out = seqmix.rglru_scan(u, self.gate_weight, self.gate_bias, self.lam, y_pre, pb, state, self.decay_scale)
        return self.out_proj(unpacked_tokens(out, s, b))
