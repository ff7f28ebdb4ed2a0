"""Laruzen: config.json -> plan.

The layers come one by one from the configuration, each a `sandwich` block (one float residual stream, an RMS norm with a gain
stored around zero before and after each sublayer, a token shift in front of the mixer, parts/sandwich.py) around one of three
mixers:

  type `gla`        `gated_linear_attention` (parts/linear_attention.py): a matrix state per head, a decay per key channel
                    through a low-rank projection;
  type `lightning`  `lightning_attention` (parts/linear_attention.py): the same with one fixed decay a head;
  type `parallel`   the mixer `side_by_side` (parts/side_by_side.py) of `attention_normed` (parts/normed_attention.py: biases,
                    normed heads and values, rotation of the front by angles computed from the position, a window, a learned sink,
                    a gate an element) and `recurrent_block` (parts/recurrent.py: a gated linear recurrence behind a short
                    convolution, beside a gelu branch).

The feed-forward is `swiglu` with the tanh form of gelu (parts/mlp.py), `routed_experts` with gated SiLU experts, the softmax
over the chosen logits as weights and a shared expert (parts/moe.py), or absent.  The stream is opened by the embedding part
`pair_embedding` (parts/pair_embedding.py), whose token before is per-request state.  Tensors are named embed, bigram,
l<i>.norm1|norm1b|norm2|norm2b|shift, l<i>.mix.<name> (l<i>.mix.left.<name>, l<i>.mix.right.<name>, l<i>.mix.left.out,
l<i>.mix.right.out), l<i>.mlp.<name> (l<i>.mlp.e<j>.<name>, l<i>.mlp.shared.<name>), final.norm, head.
"""
from __future__ import annotations

from ..config.model_config import LaruzenConfig
from ..parts.base import PartSpec
from .plan import ExecStep, ModelPlan

NO_POSITION_LIMIT = 1 << 30     # angles are computed from the position: nothing but int32 bounds it

_GATED = ("gate", "up", "down")


def _left(m: dict, D: int, eps: float, p: str, positions: dict) -> PartSpec:
    rot, position = m.get("rot") or {}, None
    if int(rot.get("dims") or 0) > 0:
        position = p + "rot"
        positions[position] = PartSpec("rope", dict(head_dim=int(m["dim"]), rotary_dim=int(rot["dims"]), max_position=NO_POSITION_LIMIT,
                                                    theta=float(rot["base"]), interleaved=False, scaling=rot.get("scaling"),
                                                    table=False, precise=True))
    return PartSpec("attention_normed", dict(hidden_size=D, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                                             dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), eps=eps, prefix=p,
                                             window=int((m.get("mask") or {}).get("size") or 0), position=position))


def _mixer(layer, D: int, eps: float, p: str, positions: dict) -> PartSpec:
    m = layer.mixer
    if layer.type == "parallel":
        r = m["right"]
        right = PartSpec("recurrent_block", dict(hidden_size=D, width=int(r["width"]), blocks=int(r["blocks"]), taps=int(r["conv"]),
                                                 prefix=p + "right."))
        return PartSpec("side_by_side", dict(left=_left(m["left"], D, eps, p + "left.", positions), right=right, hidden_size=D, eps=eps,
                                             left_norm=p + "left.out", right_norm=p + "right.out"))
    sizes = dict(hidden_size=D, num_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), eps=eps, prefix=p)
    if layer.type == "lightning":
        return PartSpec("lightning_attention", dict(sizes, decay=[float(d) for d in m["decay"]]))
    # the low-rank decay's inner size is a size of the checkpoint's tensors (-1), unless the configuration states it (a model with
    # random weights has no tensors to count)
    return PartSpec("gated_linear_attention", dict(sizes, tau=float(m["tau"]), rank=int(m.get("rank") or -1)))


def _feed_forward(mlp, D: int, p: str):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(hidden_size=D, intermediate_size=int(mlp["ff"]), prefix=p, names=_GATED, activation="gelu_tanh"))
    r, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", dict(
        hidden_size=D, expert_size=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), prefix=p,
        activation="silu_gated", scores="softmax", correction=False, normalise=True,
        shared=dict(intermediate_size=int(shared["ff"]), prefix=p + "shared.", names=_GATED) if shared else None))


def laruzen_plan(cfg: LaruzenConfig) -> ModelPlan:
    D = cfg.width
    norm = lambda name: PartSpec("rmsnorm_stream", dict(size=D, eps=cfg.eps, weight_name=name, one_plus=True))
    layers, positions = [], {}
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ff = _feed_forward(layer.mlp, D, p + "mlp.")
        layers.append(PartSpec("sandwich", dict(
            mixer=_mixer(layer, D, cfg.eps, p + "mix.", positions), feed_forward=ff, pre_mixer_norm=norm(p + "norm1"),
            post_mixer_norm=norm(p + "norm1b"), pre_ff_norm=norm(p + "norm2") if ff else None,
            post_ff_norm=norm(p + "norm2b") if ff else None, size=D, shift=p + "shift")))
    pair = {}
    if cfg.bigram is not None:
        buckets, mul_prev, mul_cur = cfg.bigram
        pair = dict(pair_name="bigram", buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_position=NO_POSITION_LIMIT,
        embedding_name="embed", lm_head_name="head", final_norm=norm("final.norm"), positions=positions, layers=layers,
        order=[ExecStep(i, i, True) for i in range(len(cfg.layers))], eos_token_id=None, default_dtype=cfg.torch_dtype,
        embedding=PartSpec("pair_embedding", dict(vocab_size=cfg.vocab, size=D, table_name="embed", **pair)))
