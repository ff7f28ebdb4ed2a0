"""Grouped-query attention with normed heads: biases, an RMS norm a head on q and k, a partial rotation with stretched
frequencies, values divided by their own root mean square, a learned sink a head, a window, a gate an element.

    q, k, v = W_q x + b_q, W_k x + b_k, W_v x + b_v                 query head h reads key/value head h / (heads / kv_heads)
    q, k    = RMSNorm_dim(q) * q.norm,  RMSNorm_dim(k) * k.norm     one gain for all heads; then the rotation of the front
    v       = v / sqrt(mean(v^2) + eps)                             (`value_norm`; no gain; cached so)
    weights = exp(s) / (exp(sink_h) + sum exp(s)),  s = (q . k) * scale       (`sink`; else the plain softmax)
    out     = W_o [ heads * sigmoid(W_g x) ] + b_o                  (`gate`: element by element)

`softcap` > 0: s becomes softcap * tanh(s / softcap).

Every option is a parameter.  q, k, v and the gate are one product; biases, norms, rotation and the cache write are one kernel
(`kernels.headnorm_rope_kv_write`).  A window lets the cache manager give back the pages behind it.  `out_bias` can be left to
the kernel that reads the output (`defer_bias`), as the pair of mixers side by side does.

The tensor-core attention kernels hold ONE head size, a multiple of 16: on the bfloat16 path a layer whose dim and vdim differ
(or are no multiple of 16) pads every head with zeros to one size when the weights are loaded (as parts/capped_attention.py).
Tensors: <prefix>q, k, v, o (+ q.b, k.b, v.b, o.b; q.norm, k.norm; sink; g).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .attention import paged_attend
from .base import NO_ROTATION, CacheSpec, Mixer, register_part
from .capped_attention import _pad_heads
from .linear import linear, linear_end
from .linear_attention import merged_rows


# Whether bfloat16 layers pad their heads to one size that the tensor-core kernels take (else such layers run the plain kernel).
PAD_HEADS = True


class NormedAttention(Mixer):
    graph_safe = True
    takes_stream_end = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float, eps: float, prefix: str,
                 positions: dict, dtype, device, window: Optional[int] = None, position: Optional[str] = None, bias: bool = True,
                 qk_norm: bool = True, value_norm: bool = True, sink: bool = True, gate: bool = True,
                 softcap: float = 0.0, **_):
        if num_heads % num_kv_heads:
            raise ValueError(f"num_heads {num_heads} is not a multiple of num_kv_heads {num_kv_heads}")
        if not 0 < dim <= 512 or not 0 < vdim <= 512:
            raise ValueError(f"head sizes dim {dim} / vdim {vdim} are not supported by the attention kernels (up to 512)")
        self.H, self.nh, self.kvh, self.kd, self.vd = int(hidden_size), int(num_heads), int(num_kv_heads), int(dim), int(vdim)
        self.scale, self.eps, self.prefix, self.window = float(scale), float(eps), prefix, int(window or 0)
        self.softcap = float(softcap or 0.0)
        self.bias, self.qk_norm, self.value_norm, self.sink, self.gate = bool(bias), bool(qk_norm), bool(value_norm), bool(sink), bool(gate)
        if position is not None and position not in positions:
            raise KeyError(f"the plan names position encoding {position!r}, but has only {sorted(positions)}")
        self.rotation = positions[position].rotation_rule() if position is not None else NO_ROTATION
        if self.rotation.rotary_dim > self.kd:
            raise ValueError(f"the position rule rotates {self.rotation.rotary_dim} dimensions, a head has {self.kd}")
        self.dtype, self.device = dtype, device
        # kp, vp: a head's size as the product writes it and the cache holds it
        one = (max(self.kd, self.vd) + 15) // 16 * 16
        padded = (PAD_HEADS and dtype == torch.bfloat16 and (self.kd != self.vd or self.kd % 16)
                  and kernels.has_fast_attention(dtype, one, self.nh // self.kvh) and self.scale > 0.0)
        self.kp, self.vp = (one, one) if padded else (self.kd, self.vd)
        self.gate_off = self.width = 0
        self.w_in = self.wo = self.b_in = self.out_bias = self.wq_norm = self.wk_norm = self.sinks = None
        self._pairs = None

    def tensor_specs(self) -> List[TensorSpec]:
        p, D, q, k, v, o = self.prefix, self.H, self.nh * self.kd, self.kvh * self.kd, self.kvh * self.vd, self.nh * self.vd
        specs = [TensorSpec(p + "q", (q, D), "matrix", D), TensorSpec(p + "k", (k, D), "matrix", D),
                 TensorSpec(p + "v", (v, D), "matrix", D), TensorSpec(p + "o", (D, o), "matrix", o)]
        if self.bias:
            specs += [TensorSpec(p + n + ".b", (c,), "coefficient", init="small") for n, c in (("q", q), ("k", k), ("v", v), ("o", D))]
        if self.qk_norm:
            specs += [TensorSpec(p + "q.norm", (self.kd,), "norm"), TensorSpec(p + "k.norm", (self.kd,), "norm")]
        if self.sink:
            specs.append(TensorSpec(p + "sink", (self.nh,), "coefficient", init="normal"))
        if self.gate:
            specs.append(TensorSpec(p + "g", (o, D), "matrix", D))
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p, kd, kp, vd, vp = self.prefix, self.kd, self.kp, self.vd, self.vp
        qkv = [_pad_heads(tensors[p + "q"], kd, kp), _pad_heads(tensors[p + "k"], kd, kp), _pad_heads(tensors[p + "v"], vd, vp)]
        parts = [torch.cat(qkv, dim=0)] + ([_pad_heads(tensors[p + "g"], vd, vp)] if self.gate else [])
        self.w_in, offs = merged_rows(parts)
        self.gate_off, self.width = (offs[1] if self.gate else 0), self.w_in.shape[0]
        self.wo = _pad_heads(tensors[p + "o"], vd, vp, dim=1).contiguous()
        if self.bias:
            self.b_in = torch.cat([_pad_heads(tensors[p + "q.b"], kd, kp), _pad_heads(tensors[p + "k.b"], kd, kp),
                                   _pad_heads(tensors[p + "v.b"], vd, vp)]).contiguous()
            self.out_bias = tensors[p + "o.b"].contiguous()
        if self.qk_norm:
            self.wq_norm, self.wk_norm = (_pad_heads(tensors[p + n], kd, kp).contiguous() for n in ("q.norm", "k.norm"))
        self.sinks = tensors[p + "sink"].contiguous() if self.sink else None
        if self.wo.is_cuda:
            self._pairs = kernels.decode_pairs_counter(self.wo.device)

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(self.kvh, self.kp, self.window, value_dim=self.vp)

    def forward(self, x, ctx, cache, state=None, write_cache: bool = True, defer_bias: bool = False, end=None):
        T = x.shape[0]
        row = linear(x, self.w_in, ctx.ws.get("normed_attn_in", T, self.width, x.dtype), ctx)
        kernels.headnorm_rope_kv_write(row, self.b_in, ctx.positions, ctx.slot_mapping[cache.group], self.wq_norm, self.wk_norm,
                                       self.rotation, cache.k, cache.v, T, self.nh, self.kvh, self.kp, self.eps, self.value_norm,
                                       write_cache, ctx.err, kd_norm=self.kd, vd_norm=self.vd)
        heads = ctx.ws.get("normed_attn_heads", T, self.nh * self.vp, x.dtype)
        paged_attend(row, self.width, heads, cache.k, cache.v, cache.group, ctx, T, self.nh, self.kvh, self.kp, self.window,
                     self.scale, self._pairs, sink=self.sinks if self.sink else False, softcap=self.softcap)
        if self.gate:
            kernels.sigmoid_gate_mul(heads, row[:, self.gate_off:], self.nh * self.vp)
        out = linear_end(heads, self.wo, ctx.ws.get("normed_attn_proj", T, self.H, x.dtype), ctx, end if self.out_bias is None else None)
        if self.out_bias is not None and not defer_bias:
            kernels.add_bias(out, self.out_bias)
        return out


register_part("mixer", "attention_normed", NormedAttention)
