"""One float residual stream with a norm in front of every sublayer, and the norm that has no statistics.

    x <- x + mixer(N1(x));   x <- x + feed_forward(N2(x))        (feed_forward None: the first line only)

The stream is float on both paths and lives in one workspace buffer [tokens, width]; it is never rounded to 16 bits.  One
kernel adds the output of the sublayer before into the stream and forms the input of the next sublayer, so a sublayer costs
one pass over the stream.  Between blocks the convention of the other blocks holds: `(hidden, residual)` = (the last
sublayer's output, not yet in the stream; the stream).

The block takes any norm that is fused with a float stream's update (`layernorm_stream`, `rmsnorm_parallel_stream` of
parts/parallel.py, or the one below).

A norm without row statistics can be made where the stream is written: in front of a `StreamTanhNorm` the block offers its
sublayer a `StreamEnd`, and a part whose last kernel can (the weight-streaming product of steps of up to 16 tokens, the sum of the
experts' rows at any size) adds into the stream and leaves the normed row behind itself.  (hidden None between blocks: nothing is
pending; `ctx.prenormed`: the next block's normed rows.)

`StreamTanhNorm`: tanh(alpha * x) * w + b with ONE learned number alpha (<weight>.alpha) and a bias (<weight>.b): no mean, no
variance, every element for itself (Zhu, Chen, He, LeCun and Liu, "Transformers without Normalization").
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Block, Norm, PartSpec, StreamEnd, build_part, register_part
from .parallel import StreamLayerNorm, StreamRMSNorm


class StreamTanhNorm(Norm):
    """tanh(alpha * x) * w + b on a float residual stream, fused with the stream's update."""
    graph_safe = True

    def __init__(self, size: int, weight_name: str, **_):
        self.size, self.weight_name = int(size), weight_name
        self.weight = self.bias = self.alpha = None

    def tensor_specs(self) -> List[TensorSpec]:
        n = self.weight_name
        return [TensorSpec(n, (self.size,), "norm"), TensorSpec(n + ".b", (self.size,), "coefficient", init="small"),
                TensorSpec(n + ".alpha", (), "coefficient", init="one")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.weight_name
        self.weight, self.bias = tensors[n].contiguous(), tensors[n + ".b"].contiguous()
        self.alpha = tensors[n + ".alpha"].reshape(1).contiguous()

    def enter(self, hidden, stream, ctx, name: str, rows=None, n_rows=None):
        """The pending outputs (`hidden` and `ctx.pending_second`) go into `stream` (None: the stream begins with `hidden`), and
        this norm of the result is returned with the stream."""
        init = stream is None
        second = None if init else getattr(ctx, "pending_second", None)
        T = hidden.shape[0] if hidden is not None else stream.shape[0]
        dtype = hidden.dtype if hidden is not None else ctx.ws.dtype
        if init:
            stream = ctx.ws.get("residual_stream", T, self.size, torch.float32)
        out = ctx.ws.get(name, T if rows is None else n_rows, self.size, dtype)
        kernels.tanh_norm_step(stream, ctx.err, y1=hidden, y2=second, alpha=self.alpha, w=self.weight, b=self.bias, out=out, rows=rows,
                               n_out=n_rows, init=init)
        if rows is None:
            ctx.pending_second = None
        return out, stream

    def forward(self, x, residual, ctx, rows=None, n_rows=None, name="normed"):
        """As a model's last norm: norm(stream after the pending writes), on the wanted rows."""
        return self.enter(x, residual, ctx, name, rows=rows, n_rows=n_rows)


# Whether sublayers may end in the stream themselves (else the stream's step is always a kernel of its own).
END_IN_STREAM = True


class PreNormStreamBlock(Block):
    def __init__(self, mixer: PartSpec, feed_forward: Optional[PartSpec], input_norm: PartSpec, post_mixer_norm: Optional[PartSpec],
                 size: int, **common):
        self.size = int(size)
        self.input_norm = build_part("norm", input_norm, **common)
        self.mixer = build_part("mixer", mixer, **common)
        self.feed_forward = build_part("feed_forward", feed_forward, **common) if feed_forward is not None else None
        self.post_mixer_norm = build_part("norm", post_mixer_norm, **common) if feed_forward is not None else None
        for n in (self.input_norm, self.post_mixer_norm):
            if n is not None and not isinstance(n, (StreamTanhNorm, StreamLayerNorm, StreamRMSNorm)):
                raise ValueError("the block fuses its norms into the stream's kernel: they must be of kind 'tanh_stream', "
                                 "'layernorm_stream' or 'rmsnorm_parallel_stream'")
        self._parts = [p for p in (self.input_norm, self.mixer, self.post_mixer_norm, self.feed_forward) if p is not None]
        self.graph_safe = all(p.graph_safe for p in self._parts)

    def parts(self):
        return list(self._parts)

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self._parts for s in p.tensor_specs()]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self._parts:
            p.load({s.name: tensors[s.name] for s in p.tensor_specs()})

    def _offer(self, part, norm, normed, stream, ctx) -> dict:
        """The `end` argument of a sublayer that reads `normed` and is followed by `norm` (None: by nothing)."""
        if not END_IN_STREAM or not part.takes_stream_end or not (norm is None or isinstance(norm, StreamTanhNorm)):
            return {}
        out = None
        if norm is not None:        # the other of the two buffers: the sublayer's own input is not written over
            out = next(b for b in (ctx.ws.get(n, normed.shape[0], self.size, normed.dtype) for n in ("normed", "normed_ff"))
                       if b.data_ptr() != normed.data_ptr())
        return dict(end=StreamEnd(stream, norm, out))

    def forward(self, hidden, residual, ctx, cache, state, write_cache=True):
        ahead, ctx.prenormed = getattr(ctx, "prenormed", None), None
        if hidden is None and isinstance(ahead, StreamEnd) and ahead.norm is self.input_norm:
            normed, stream = ahead.normed, residual
        else:
            normed, stream = self.input_norm.enter(hidden, residual, ctx, "normed")
        following = getattr(ctx, "next_norm", None)
        offer = self._offer(self.mixer, following if self.feed_forward is None else self.post_mixer_norm, normed, stream, ctx)
        y = self.mixer.forward(normed, ctx, cache, state, write_cache, **offer)
        if self.feed_forward is not None:
            if y is None:
                normed = offer["end"].normed
            else:
                normed, stream = self.post_mixer_norm.enter(y, stream, ctx, "normed_ff")
            offer = self._offer(self.feed_forward, following, normed, stream, ctx)
            y = self.feed_forward.forward(normed, ctx, **offer)
        if y is None:
            ctx.prenormed = offer["end"]
        return y, stream


def stream_value(hidden, stream, ctx) -> torch.Tensor:
    """The residual stream [tokens, width] (float, a new tensor) after the pending write of `hidden`: what the next norm would
    see.  For inspection; no step of the engine needs it."""
    x = stream.clone()
    if hidden is None and getattr(ctx, "pending_second", None) is None:
        return x
    kernels.tanh_norm_step(x, ctx.err, y1=hidden, y2=getattr(ctx, "pending_second", None))
    return x


register_part("norm", "tanh_stream", StreamTanhNorm)
register_part("block", "pre_norm_stream", PreNormStreamBlock)
