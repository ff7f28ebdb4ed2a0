"""Linear attention as token mixers: a matrix state per head with a decay, no correction of what is written.

`GatedLinearAttention`, a decay per key channel that the input decides:

    q = W_q x * dim^(-1/2),  k = W_k x  [heads, dim],   v = W_v x  [heads, vdim]
    alpha = sigmoid(W_a2 (W_a1 x) + b)^(1 / tau)         [heads, dim]
    S <- diag(alpha) S + k v^T,   o = S^T q              per head, S [dim, vdim]
    out = W_o [ RMSNorm_vdim(o) * norm * SiLU(W_g x) ]   norm: one weight for all heads

(Yang, Wang, Shen, Panda and Kim, "Gated Linear Attention Transformers with Hardware-Efficient Training".)

`LightningAttention`, one fixed decay a head:

    q = SiLU(W_q x),  k = SiLU(W_k x),  v = SiLU(W_v x);   S <- decay_h S + k v^T,   o = S^T q
    out = W_o [ RMSNorm(o over all heads) * norm * sigmoid(W_g x) ]

`MLSTM`, a matrix memory with exponential gates held in range by a running maximum (Beck, Poeppel, Spanring and others, "xLSTM:
Extended Long Short-Term Memory"), its log gates soft-capped:

    q = W_q x * dim^(-1/2),  k = W_k x  [heads, dim],   v = W_v x  [heads, vdim]
    i = cap * tanh((W_i x + b_i) / cap),   f = log sigmoid(cap * tanh((W_f x + b_f) / cap))        one of each a head
    m <- max(f + m, i);   S <- exp(f + m' - m) S + exp(i - m) k v^T,   n likewise with k alone     (m' the maximum before; all 0 first)
    o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
    out = W_o [ RMSNorm_vdim(o) * norm * sigmoid(W_g x) ]                                          norm: a gain an element of every head

Its state is the matrices, behind them n [heads, dim] and m [heads]; the gates of a portion are made ahead of its walk, from a scan of
the maxima over the tokens.

All projections of x are one product.  The state, [heads, dim, vdim] floats a request, lives in the cache manager's state slots;
decays, their logarithms, the recurrence and the norms are float on both paths.  The walks are those of the package's other
matrix states with a gate a row (csrc/kernels/recurrent.cu): one block a (request, head) while decoding, columns over blocks
and long portions cut along the tokens otherwise.
"""
from __future__ import annotations

from typing import Dict, List, Sequence

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Mixer, StateSpec, register_part
from .linear import linear, linear_end


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def merged_rows(parts: Sequence[torch.Tensor]):
    """The rows of several matrices over the same input as one matrix, each starting at a multiple of 8 (so that every part of a
    projected row starts on a 16-byte boundary), and where each starts."""
    rows, offs, at = [], [], 0
    for w in parts:
        offs.append(at)
        rows.append(w)
        pad = _up8(w.shape[0]) - w.shape[0]
        if pad:
            rows.append(w.new_zeros((pad, w.shape[1])))
        at += w.shape[0] + pad
    return torch.cat(rows, dim=0).contiguous(), offs


class _MatrixState(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, eps: float, prefix: str):
        self.H, self.nh, self.dk, self.dv = int(hidden_size), int(num_heads), int(dim), int(vdim)
        self.eps, self.prefix = float(eps), prefix
        if self.dk > 256:
            raise ValueError(f"the scan keeps a column of the state in registers: dim up to 256, not {self.dk}")
        self.w_in = self.wo = self.norm_weight = None
        self.gate_off = 0

    def _projections(self) -> List[TensorSpec]:
        p, H, qd, vd = self.prefix, self.H, self.nh * self.dk, self.nh * self.dv
        return [TensorSpec(p + "q", (qd, H), "matrix", H), TensorSpec(p + "k", (qd, H), "matrix", H),
                TensorSpec(p + "v", (vd, H), "matrix", H), TensorSpec(p + "g", (vd, H), "matrix", H),
                TensorSpec(p + "o", (H, vd), "matrix", vd)]

    def _qkv(self, tensors) -> torch.Tensor:
        return torch.cat([tensors[self.prefix + n] for n in ("q", "k", "v")], dim=0)

    def state_spec(self) -> StateSpec:
        return StateSpec((self.nh * self.dk * self.dv,), torch.float32)

    def _chunks(self, T: int, ctx, extra: int = 0):
        """Ranges a request's tokens are cut into, and the scratch they need (`extra`: columns beside a head's dv)."""
        B = ctx.launch_requests
        chunks = kernels.matrix_scan_chunks(T, B, self.nh, self.dk, self.dv)
        scratch = None if chunks == 1 else ctx.ws.get_flat("matrix_scan_ranges", B * chunks * self.nh * self.dk * (self.dv + 1 + extra),
                                                           torch.float32)
        return chunks, scratch


class GatedLinearAttention(_MatrixState):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, tau: float, eps: float, prefix: str, rank: int = -1,
                 dtype=None, device=None, **_):
        """`rank` -1: the low-rank decay's inner size is read from the checkpoint's tensors."""
        super().__init__(hidden_size, num_heads, dim, vdim, eps, prefix)
        self.tau, self.rank = float(tau), int(rank)
        self.w_a2 = self.bias = None
        self.a_off = self.a_pad = self.z_off = self.width1 = self.width = 0

    def tensor_specs(self) -> List[TensorSpec]:
        p, H, qd, r = self.prefix, self.H, self.nh * self.dk, self.rank
        return self._projections() + [TensorSpec(p + "a1", (r, H), "matrix", H), TensorSpec(p + "a2", (qd, r), "matrix", max(r, 1)),
                                      TensorSpec(p + "a2.b", (qd,), "coefficient", init="normal"),
                                      TensorSpec(p + "norm", (self.dv,), "norm")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        a1, a2 = tensors[p + "a1"], tensors[p + "a2"]
        self.rank = int(a1.shape[0])
        if a2.shape[1] != self.rank:
            raise ValueError(f"{p}a2 has {a2.shape[1]} columns for the {self.rank} rows of {p}a1")
        # 16-bit decode steps: the inner size in whole groups of 64, as the weight-streaming product takes it (zeros behind)
        self.a_pad = (self.rank + 63) // 64 * 64 if a1.dtype == torch.bfloat16 else self.rank
        wide1, wide2 = a1.new_zeros((self.a_pad, self.H)), a2.new_zeros((a2.shape[0], self.a_pad))
        wide1[:self.rank], wide2[:, :self.rank] = a1, a2
        self.w_in, (_, self.gate_off, self.a_off) = merged_rows([self._qkv(tensors), tensors[p + "g"], wide1])
        self.w_a2, self.bias = wide2.contiguous(), tensors[p + "a2.b"].contiguous()
        self.width1 = self.z_off = self.w_in.shape[0]
        self.width = self.z_off + _up8(self.nh * self.dk)
        self.norm_weight, self.wo = tensors[p + "norm"].contiguous(), tensors[p + "o"].contiguous()

    def forward(self, x, ctx, cache, state, write_cache: bool = True):
        T, B = x.shape[0], ctx.launch_requests
        row = ctx.ws.get("gla_in", T, self.width, x.dtype)
        linear(x, self.w_in, row[:, :self.width1], ctx)
        linear(row[:, self.a_off:self.a_off + self.a_pad], self.w_a2, row[:, self.z_off:self.z_off + self.nh * self.dk], ctx)
        out = ctx.ws.get("gla_out", T, self.nh * self.dv, x.dtype)
        common = (row, self.z_off, self.gate_off, self.bias, self.norm_weight, state, ctx.cu_q, ctx.state_slots, B, self.nh, self.dk,
                  self.dv, self.dk ** -0.5, self.tau, self.eps, ctx.err)
        single = ctx.max_q <= 1
        if kernels.matrix_scan_fuses(self.dk, self.dv, T, B, single):
            kernels.gla_scan(*common, out=out, single=single)
        else:
            raw = ctx.ws.get("matrix_scan_raw", T, self.nh * self.dv, torch.float32)
            chunks, scratch = self._chunks(T, ctx)
            kernels.gla_scan(*common, raw=raw, chunks=chunks, scratch=scratch)
            kernels.delta_out_norm(raw, row[:, self.gate_off:], self.norm_weight, out, T, self.nh, self.dv, self.eps)
        return linear(out, self.wo, ctx.ws.get("mixer_proj", T, self.H, x.dtype), ctx)


class LightningAttention(_MatrixState):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float, prefix: str,
                 dtype=None, device=None, **_):
        super().__init__(hidden_size, num_heads, dim, vdim, eps, prefix)
        if len(decay) != self.nh:
            raise ValueError(f"{len(decay)} decays for {self.nh} heads")
        self.decay, self.decays = [float(d) for d in decay], None

    def tensor_specs(self) -> List[TensorSpec]:
        return self._projections() + [TensorSpec(self.prefix + "norm", (self.nh * self.dv,), "norm")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        self.w_in, (_, self.gate_off) = merged_rows([self._qkv(tensors), tensors[p + "g"]])
        self.norm_weight, self.wo = tensors[p + "norm"].contiguous(), tensors[p + "o"].contiguous()
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=self.wo.device)

    def forward(self, x, ctx, cache, state, write_cache: bool = True):
        T, B = x.shape[0], ctx.launch_requests
        row = linear(x, self.w_in, ctx.ws.get("lightning_in", T, self.w_in.shape[0], x.dtype), ctx)
        raw = ctx.ws.get("matrix_scan_raw", T, self.nh * self.dv, torch.float32)
        chunks, scratch = self._chunks(T, ctx)
        kernels.lightning_scan(row, self.decays, state, ctx.cu_q, ctx.state_slots, raw, B, self.nh, self.dk, self.dv, ctx.err,
                               chunks=chunks, scratch=scratch, single=ctx.max_q <= 1 and kernels.matrix_scan_fuses(self.dk, self.dv, T, B, True))
        out = ctx.ws.get("lightning_out", T, self.nh * self.dv, x.dtype)
        # one norm over all heads: a row is one "head" of heads * vdim elements
        kernels.delta_out_norm(raw, row[:, self.gate_off:], self.norm_weight, out, T, 1, self.nh * self.dv, self.eps, gate_sigmoid=True)
        return linear(out, self.wo, ctx.ws.get("mixer_proj", T, self.H, x.dtype), ctx)


class MLSTM(_MatrixState):
    takes_stream_end = True

    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, gate_cap: float, eps: float, prefix: str, dtype=None,
                 device=None, **_):
        super().__init__(hidden_size, num_heads, dim, vdim, eps, prefix)
        self.cap = float(gate_cap)
        if not self.cap > 0.0:
            raise ValueError(f"the cap of the gates must be positive, not {gate_cap}")
        self.bias_i = self.bias_f = None
        self.i_off = self.f_off = 0

    def tensor_specs(self) -> List[TensorSpec]:
        p, H, nh = self.prefix, self.H, self.nh
        return self._projections() + [TensorSpec(p + "i", (nh, H), "matrix", H), TensorSpec(p + "i.b", (nh,), "coefficient", init="small"),
                                      TensorSpec(p + "f", (nh, H), "matrix", H), TensorSpec(p + "f.b", (nh,), "coefficient", init="open"),
                                      TensorSpec(p + "norm", (nh * self.dv,), "norm")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p = self.prefix
        gates = torch.cat([tensors[p + "i"], tensors[p + "f"]], dim=0)
        self.w_in, (_, self.gate_off, self.i_off) = merged_rows([self._qkv(tensors), tensors[p + "g"], gates])
        self.f_off = self.i_off + self.nh
        self.bias_i, self.bias_f = tensors[p + "i.b"].contiguous(), tensors[p + "f.b"].contiguous()
        self.norm_weight, self.wo = tensors[p + "norm"].contiguous(), tensors[p + "o"].contiguous()

    def state_spec(self) -> StateSpec:
        n = self.nh * (self.dk * (self.dv + 1) + 1)
        return StateSpec(((n + 3) // 4 * 4,), torch.float32)      # rows stay 16-byte aligned

    def forward(self, x, ctx, cache, state, write_cache: bool = True, end=None):
        T, B, nh, dk, dv = x.shape[0], ctx.launch_requests, self.nh, self.dk, self.dv
        row = linear(x, self.w_in, ctx.ws.get("mlstm_in", T, self.w_in.shape[0], x.dtype), ctx)
        out = ctx.ws.get("mlstm_out", T, nh * dv, x.dtype)
        common = (row, self.i_off, self.f_off, self.gate_off, self.bias_i, self.bias_f, self.norm_weight, state, ctx.cu_q,
                  ctx.state_slots, B, nh, dk, dv, dk ** -0.5, self.cap, self.eps, ctx.err)
        single = ctx.max_q <= 1
        if kernels.matrix_scan_fuses(dk, dv, T, B, single):
            kernels.mlstm_scan(*common, out=out, single=single)
        else:
            gates = ctx.ws.get("mlstm_gates", T, nh * 4, torch.float32)
            raw = ctx.ws.get("matrix_scan_raw", T, nh * dv, torch.float32)
            nq = ctx.ws.get("mlstm_normaliser", T, nh, torch.float32)
            chunks, scratch = self._chunks(T, ctx, extra=1)
            kernels.mlstm_scan(*common, gates=gates, raw=raw, nq=nq, chunks=chunks, scratch=scratch)
            kernels.delta_out_norm(raw, row[:, self.gate_off:], self.norm_weight, out, T, nh, dv, self.eps, gate_sigmoid=True, nq=nq,
                                   gates=gates)
        return linear_end(out, self.wo, ctx.ws.get("mixer_proj", T, self.H, x.dtype), ctx, end)


register_part("mixer", "mlstm", MLSTM)
register_part("mixer", "gated_linear_attention", GatedLinearAttention)
register_part("mixer", "lightning_attention", LightningAttention)
