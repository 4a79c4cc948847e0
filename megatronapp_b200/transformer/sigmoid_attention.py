"""Grouped-query attention whose weights are logistic functions of the scores, with rotary queries, keys and values.

Per token at position ``i``, from the mixer input ``x``::

    q, k = rms_norm_per_head(R_i W_q x), rms_norm_per_head(R_i W_k x)        R_i: rotation by the position, no norm weight
    v    = V_i W_v x                                                         V_i: rotation of the whole value
    s_j  = cap(q_h . k_kv(h)(j) * scale) + bias_h,   j <= i;   cap(z) = softcap tanh(z / softcap)
    o_h  = V_i^-1 sum_j sigmoid(s_j) v_kv(h)(j);   y = W_o concat(o)

The weights are not normalised over the keys (Ramapuram et al., "Theory, Analysis, and Best Practices for Sigmoid
Self-Attention").  Because values are turned by their own position before they are cached and the sum is turned back by the
query's, a value enters by its distance.  Pairs are ``(i, i + n)`` or ``interleaved``; values share the layout and the base.

The module follows the framework's other paged mixers: one fused input projection ``[q | k | v]``, rotated and normed keys
and rotated values in the paged cache of the inference context, a row-parallel output projection.  Angles, norm statistics,
scores, weights and the weighted sum are fp32.  A step in which every sequence starts (fresh prompts) has all its keys at
hand: with 16-bit activations and heads of at most 128 it runs through the tcgen05 kernel (``ops.sigmoid_attention``), the
head operands padded to the kernel's width by the rotation kernel that writes them.  Every size and constant is a parameter.
"""
from __future__ import annotations

import os
from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..ops import seqmix
from ..ops.seqmix import HeadPart
from ..parallel.tp_layers import ColumnParallelLinear, RowParallelLinear
from ..ssm.gated_delta import packed_tokens, unpacked_tokens
from .mixed_head_attention import dense_pages
from .module import MegatronModule


class SigmoidAttention(MegatronModule):
    FLASH_PREFILL_MIN_TOKENS = 64

    def __init__(self, config, layer_number: int, num_heads: int, num_kv_heads: int, qk_dim: int, v_dim: int, scale: float,
                 softcap: float = 0.0, rot_dims: int = 0, rot_base: float = 10000.0, rot_scaling: Optional[dict] = None,
                 interleaved: bool = False, rotate_values: bool = True, qk_norm: bool = True, eps: Optional[float] = None):
        super().__init__(config)
        if num_heads % num_kv_heads:
            raise ValueError("sigmoid attention: heads must be a multiple of kv_heads")
        if rot_dims % 2 or rot_dims > qk_dim:
            raise ValueError("sigmoid attention: rot_dims must be even and at most the head dimension")
        if rotate_values and v_dim % 2:
            raise ValueError("sigmoid attention: rotated values need an even value dimension")
        self.layer_number = layer_number
        self.nh, self.nkv, self.d, self.dv = num_heads, num_kv_heads, qk_dim, v_dim
        self.scale, self.softcap, self.interleaved, self.qk_norm = float(scale), float(softcap), bool(interleaved), bool(qk_norm)
        self.eps = config.layernorm_epsilon if eps is None else eps
        self.q_ch, self.k_ch, self.v_ch = num_heads * qk_dim, num_kv_heads * qk_dim, num_kv_heads * v_dim
        self.in_proj = ColumnParallelLinear(config.hidden_size, self.q_ch + self.k_ch + self.v_ch, config=config,
                                            init_method=config.init_method, bias=False, skip_bias_add=False, gather_output=False)
        dev, dt_ = self.in_proj.weight.device, config.params_dtype
        self.head_bias = nn.Parameter(torch.zeros(num_heads, device=dev, dtype=dt_))
        turns, self.amplitude = seqmix.rotary_turns(rot_dims, rot_base, rot_scaling, dev)
        self.register_buffer("turns", turns, persistent=False)
        self.register_buffer("value_turns", seqmix.rotary_turns(v_dim, rot_base, None, dev)[0] if rotate_values else None, persistent=False)
        self.out_proj = RowParallelLinear(num_heads * v_dim, config.hidden_size, config=config, init_method=config.output_layer_init_method,
                                          bias=False, input_is_parallel=True, skip_bias_add=True)

    def segments(self):
        """Row counts of the ``[q | k | v]`` segments of ``in_proj``."""
        return [("q", self.q_ch), ("k", self.k_ch), ("v", self.v_ch)]

    def _flash_prefill(self, proj, ctx) -> bool:
        return (ctx.fresh_prefill and ctx.min_new >= self.FLASH_PREFILL_MIN_TOKENS and proj.is_cuda
                and proj.dtype in (torch.bfloat16, torch.float16) and max(self.d, self.dv) <= 128
                and os.environ.get("B200_SIGMOID_FLASH_PREFILL", "1") == "1" and ops.native_attention_available())

    def forward(self, hidden_states, inference_context=None, cache_index=None, **_):
        s, b = hidden_states.shape[0], hidden_states.shape[1]
        key = self.layer_number if cache_index is None else cache_index
        proj, _ = self.in_proj(hidden_states)
        proj = packed_tokens(proj)                                                     # [T, q | k | v]
        T = proj.shape[0]
        q = proj[:, :self.q_ch].unflatten(1, (self.nh, self.d))
        k = proj[:, self.q_ch:self.q_ch + self.k_ch].unflatten(1, (self.nkv, self.d))
        v = proj[:, self.q_ch + self.k_ch:].unflatten(1, (self.nkv, self.dv))
        ctx = inference_context
        flash = False
        if ctx is not None:
            if ctx.is_static_batching():
                raise NotImplementedError("sigmoid attention serves through the dynamic (paged) engine")
            kc, vc = ctx.kv_pages(key, (self.nkv, self.d), (self.nkv, self.dv), proj.dtype)
            slots, positions = ctx.write_slots, ctx.positions
            flash = self._flash_prefill(proj, ctx)
        else:
            table, tok_req, tok_len = dense_pages(s, b, proj.device)
            kc = vc = slots = None
            positions = tok_len.long() - 1
        width = (64 if max(self.d, self.dv) <= 64 else 128) if flash else self.d
        qr = proj.new_empty(T, self.nh, width)
        kr = vr = None
        if flash or ctx is None:
            kr, vr = proj.new_empty(T, self.nkv, width), proj.new_empty(T, self.nkv, width if flash else self.dv)
        half, back = 0, None
        if flash and self.value_turns is not None:                      # what the tcgen05 kernel turns the result back by
            half = 0 if self.interleaved else width // 2
            back = torch.empty(T, self.value_turns.shape[0], 2, dtype=torch.float32, device=proj.device)
        kw = dict(turns=self.turns, interleaved=self.interleaved, amplitude=self.amplitude, rms=self.qk_norm)
        seqmix.head_rotary([HeadPart(q, out=qr, **kw), HeadPart(k, out=kr, pages=kc, **kw),
                            HeadPart(v, self.value_turns, self.interleaved, out=vr, pages=vc, out_half=half, table=back)],
                           positions, self.eps, slots)
        if flash:
            o = ops.sigmoid_attention(qr, kr, vr, ctx.packed.cu, ctx.packed.max_len, self.scale, self.softcap, self.head_bias, back,
                                      self.interleaved, self.dv)
        elif ctx is not None:
            o = ctx.attend_sigmoid(key, qr, self.scale, self.softcap, self.head_bias, self.value_turns, self.interleaved)
        else:
            o = seqmix.sigmoid_attention_paged(qr, kr, vr, table, tok_req, tok_len, s, self.scale, self.softcap, self.head_bias,
                                               self.value_turns, self.interleaved)
        return self.out_proj(unpacked_tokens(o, s, b))
