"""Recurrent token mixers: a fixed-size state per request instead of pages.

Both keep their state in float in the cache manager's state slots (`state_spec()`), carried from step to step;
a request's slot is zeroed when it is assigned.  Projections are the package's usual products (merged where several
read the same input); gates, decays and the recurrence itself are float inside one scan kernel a mixer.

`MinGRU`: both gates are functions of the current token alone, never of the state.  z = sigmoid(Wz h + bz), u = Wx h + bx, candidate = u + 1/2 where
u >= 0 and sigmoid(u) below, s_t = (1 - z) s_{t-1} + z * candidate (element by element, `width` channels), output
Wo (s_t * silu(Wg h)).  (The recurrence of Feng, Tung, Ahmed, Bengio and Hajimirsadeghi, "Were RNNs All We Needed?".)

`HGRN2`: a matrix-valued state per head with one gate for two jobs: f keeps, 1 - f writes.  Per head q = silu(Wq h) [dim],
v = Wv h [vdim], f = l + (1 - l) sigmoid(Wf h + bf) [dim] with a learned lower bound l; the state M [dim, vdim] goes
M_t = diag(f_t) M_{t-1} + (1 - f_t) v_t^T, o_t = M_t^T q_t; o is RMS-normed over vdim (a weight shared by the heads),
heads are concatenated and projected by Wo.

`RecurrentBlock`: a gated linear recurrence behind a short convolution, beside a gelu branch (the recurrent block of De, Smith,
Fernando and others, "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models").  With
`width` channels in `blocks` equal parts:

    y = gelu(Wy h + by),   u = conv(Wx h + bx) + bc          (tanh-form gelu; a causal filter a channel over time, no activation)
    r = sigmoid(ra_b u_b + br_b),  i = sigmoid(ri_b u_b + bi_b)            for every part u_b of u, ra_b and ri_b square
    log a = -8 r softplus(lam),   S_t = a S_{t-1} + sqrt(1 - a^2) i u,     output Wo (S * y)

The state is S and the last taps - 1 inputs of the filter.  u is of the model's type; the gates' products leave in float, and
gates, decays and the recurrence are float in one scan kernel that also applies the gelu branch.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Mixer, StateSpec, register_part
from .delta import SHORT_PORTIONS
from .linear import linear
from .linear_attention import merged_rows


class MinGRU(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, width: int, prefix: str, dtype=None, device=None, **_):
        self.H, self.W, self.prefix = int(hidden_size), int(width), prefix
        self.wzxg = self.wo = self.bz = self.bx = None

    def tensor_specs(self) -> List[TensorSpec]:
        p, H, W = self.prefix, self.H, self.W
        return [TensorSpec(p + "z", (W, H), "matrix", H), TensorSpec(p + "z.b", (W,), "bias"),
                TensorSpec(p + "x", (W, H), "matrix", H), TensorSpec(p + "x.b", (W,), "bias"),
                TensorSpec(p + "g", (W, H), "matrix", H), TensorSpec(p + "o", (H, W), "matrix", W)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        # rows of z, then the candidate, then the output gate: one product for the three
        self.wzxg = torch.cat([tensors[p + "z"], tensors[p + "x"], tensors[p + "g"]], dim=0).contiguous()
        self.bz, self.bx = tensors[p + "z.b"].contiguous(), tensors[p + "x.b"].contiguous()
        self.wo = tensors[p + "o"].contiguous()

    def state_spec(self) -> StateSpec:
        return StateSpec((self.W,), torch.float32)

    def forward(self, x, ctx, cache, state, write_cache: bool = True):
        T = x.shape[0]
        zxg = linear(x, self.wzxg, ctx.ws.get("mingru_zxg", T, 3 * self.W, x.dtype), ctx)
        gated = ctx.ws.get("mingru_out", T, self.W, x.dtype)
        kernels.mingru_scan(zxg, self.bz, self.bx, state, ctx.cu_q, ctx.state_slots, gated, ctx.launch_requests, ctx.err,
                            chunks=kernels.scan_chunks(T, ctx.launch_requests))
        return linear(gated, self.wo, ctx.ws.get("mixer_proj", T, self.H, x.dtype), ctx)


class HGRN2(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, eps: float, prefix: str, dtype=None,
                 device=None, **_):
        self.H, self.nh, self.dk, self.dv, self.eps, self.prefix = int(hidden_size), int(num_heads), int(dim), int(vdim), float(eps), prefix
        if self.dk > 256:
            raise ValueError(f"the HGRN2 scan keeps a column of the state in registers: dim up to 256, not {self.dk}")
        self.wqfv = self.wo = self.bf = self.lower = self.norm_weight = None

    def tensor_specs(self) -> List[TensorSpec]:
        p, H, qd, vd = self.prefix, self.H, self.nh * self.dk, self.nh * self.dv
        return [TensorSpec(p + "q", (qd, H), "matrix", H), TensorSpec(p + "f", (qd, H), "matrix", H),
                TensorSpec(p + "f.b", (qd,), "bias"), TensorSpec(p + "lower", (qd,), "coefficient", init="fraction"),
                TensorSpec(p + "v", (vd, H), "matrix", H), TensorSpec(p + "norm", (self.dv,), "norm"),
                TensorSpec(p + "o", (H, vd), "matrix", vd)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        self.wqfv = torch.cat([tensors[p + "q"], tensors[p + "f"], tensors[p + "v"]], dim=0).contiguous()
        self.bf, self.lower = tensors[p + "f.b"].contiguous(), tensors[p + "lower"].contiguous()
        self.norm_weight, self.wo = tensors[p + "norm"].contiguous(), tensors[p + "o"].contiguous()

    def state_spec(self) -> StateSpec:
        return StateSpec((self.nh, self.dk, self.dv), torch.float32)

    def forward(self, x, ctx, cache, state, write_cache: bool = True):
        T = x.shape[0]
        width = self.nh * (2 * self.dk + self.dv)
        qfv = linear(x, self.wqfv, ctx.ws.get("hgrn2_qfv", T, width, x.dtype), ctx)
        out = ctx.ws.get("hgrn2_out", T, self.nh * self.dv, x.dtype)
        # decoding: one block a (request, head), norm included; portions: a head's columns over several blocks
        single = ctx.max_q <= 1
        fuse = kernels.matrix_scan_fuses(self.dk, self.dv, T, ctx.launch_requests, single)
        raw = None if fuse else ctx.ws.get("hgrn2_raw", T, self.nh * self.dv, torch.float32)
        # longer portions are also cut along the tokens
        B = ctx.launch_requests
        chunks = 1 if fuse else kernels.matrix_scan_chunks(T, B, self.nh, self.dk, self.dv)
        scratch = None if chunks == 1 else ctx.ws.get_flat("hgrn2_ranges", B * chunks * self.nh * self.dk * (self.dv + 1),
                                                           torch.float32)
        kernels.hgrn2_scan(qfv, self.bf, self.lower, self.norm_weight, state, ctx.cu_q, ctx.state_slots, out,
                           B, self.nh, self.dk, self.dv, self.eps, ctx.err, raw=raw, chunks=chunks, scratch=scratch, single=single and fuse)
        return linear(out, self.wo, ctx.ws.get("mixer_proj", T, self.H, x.dtype), ctx)


class RecurrentBlock(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, width: int, blocks: int, taps: int, prefix: str, dtype=None, device=None, **_):
        self.H, self.W, self.blocks, self.taps, self.prefix = int(hidden_size), int(width), int(blocks), int(taps), prefix
        if self.blocks <= 0 or self.W % self.blocks:
            raise ValueError(f"{self.W} channels do not fall into {self.blocks} equal parts")
        if not 1 <= self.taps <= 9:
            raise ValueError(f"the short convolution takes 1 to 9 taps, not {self.taps}")
        self.w_in = self.wo = self.w_gates = self.conv_w = None
        self.by = self.bx = self.bc = self.br = self.bi = self.lam = None
        self.x_off = 0

    def tensor_specs(self) -> List[TensorSpec]:
        p, H, W, n, s = self.prefix, self.H, self.W, self.blocks, self.W // self.blocks
        small = lambda name, shape: TensorSpec(p + name, shape, "coefficient", init="small")
        return [TensorSpec(p + "y", (W, H), "matrix", H), small("y.b", (W,)), TensorSpec(p + "x", (W, H), "matrix", H), small("x.b", (W,)),
                TensorSpec(p + "conv", (W, self.taps), "coefficient", self.taps, init="normal"), small("conv.b", (W,)),
                TensorSpec(p + "ra", (n, s, s), "matrix", s), small("ra.b", (n, s)),
                TensorSpec(p + "ri", (n, s, s), "matrix", s), small("ri.b", (n, s)),
                TensorSpec(p + "lam", (W,), "coefficient", init="normal"), TensorSpec(p + "o", (H, W), "matrix", W)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        self.w_in, (_, self.x_off) = merged_rows([tensors[p + "y"], tensors[p + "x"]])
        # per part [in, out of r | out of i], as head_linear and the batched product read them
        self.w_gates = torch.cat([tensors[p + "ra"].transpose(1, 2), tensors[p + "ri"].transpose(1, 2)], dim=2).contiguous()
        self.conv_w = tensors[p + "conv"].contiguous()
        self.by, self.bx, self.bc = (tensors[p + n].contiguous() for n in ("y.b", "x.b", "conv.b"))
        self.br, self.bi = (tensors[p + n].reshape(self.W).contiguous() for n in ("ra.b", "ri.b"))
        self.lam, self.wo = tensors[p + "lam"].contiguous(), tensors[p + "o"].contiguous()

    def state_spec(self) -> StateSpec:
        return StateSpec((self.W * self.taps,), torch.float32)

    def forward(self, x, ctx, cache, state, write_cache: bool = True):
        T, B, W = x.shape[0], ctx.launch_requests, self.W
        row = linear(x, self.w_in, ctx.ws.get("recurrent_in", T, self.w_in.shape[0], x.dtype), ctx)
        u = ctx.ws.get("recurrent_u", T, W, x.dtype)
        branch = row[:, self.x_off:]
        if ctx.max_q <= SHORT_PORTIONS:
            kernels.short_conv_step(branch, W, self.conv_w, state, W, ctx.cu_q, ctx.state_slots, u, B, ctx.err, activation=False,
                                    bias_in=self.bx, bias_out=self.bc)
        else:
            kernels.short_conv_silu(branch, W, self.conv_w, state, W, ctx.token_req, ctx.cu_q, ctx.state_slots, u, T, ctx.err,
                                    activation=False, bias_in=self.bx, bias_out=self.bc)
            kernels.short_conv_state(branch, W, self.taps, state, W, ctx.cu_q, ctx.state_slots, B, bias_in=self.bx)
        gates = ctx.ws.get("recurrent_gates", T, 2 * W, torch.float32)
        part = W // self.blocks
        if LIBRARY_GATE_PRODUCTS and x.dtype == torch.bfloat16 and T > 16:
            torch.bmm(torch.as_strided(u, (self.blocks, T, part), (part, W, 1)), self.w_gates, out_dtype=torch.float32,
                      out=torch.as_strided(gates, (self.blocks, T, 2 * part), (2 * part, 2 * W, 1)))
        else:
            kernels.head_linear(u, W, part, self.w_gates, gates, 2 * W, 2 * part, T)
        out = ctx.ws.get("recurrent_out", T, W, x.dtype)
        kernels.lru_scan(u, gates, row, self.br, self.bi, self.lam, self.by, state, ctx.cu_q, ctx.state_slots, out, B, self.blocks,
                         ctx.err, chunks=64 if T > 1024 * B else kernels.scan_chunks(T, B))
        return linear(out, self.wo, ctx.ws.get("recurrent_proj", T, self.H, x.dtype), ctx)


# bfloat16 steps of more than 16 tokens: the gates' products of the parts go to the library's batched product with float
# results (as the package's other products of that size do); smaller steps and the 32-bit path use head_linear
LIBRARY_GATE_PRODUCTS = True

register_part("mixer", "recurrent_block", RecurrentBlock)
register_part("mixer", "mingru", MinGRU)
register_part("mixer", "hgrn2", HGRN2)
