"""Nesezen: config.json -> plan.

The layers come one by one from the configuration, each a `pre_norm_stream` block (one float residual stream, in front of each
sublayer the norm tanh(alpha x) * w + b, parts/pre_norm_stream.py) around one of three mixers:

  type `attention`         `attention_normed` (parts/normed_attention.py) with nothing normed, biased or gated: grouped queries, the
                           front of every head rotated in halves by angles computed from the position, with frequencies stretched
                           by wavelength, capped scores, a sliding window;
  type `mlstm`             `mlstm` (parts/linear_attention.py): a matrix state per head with exponential gates;
  type `latent_attention`  `latent_attention` (parts/latent_attention.py) without positions, with a gate a head.

The feed-forward is `swiglu` (parts/mlp.py), `routed_experts` (parts/moe.py: gated SiLU experts, sigmoid scores that multiply the
experts' inputs, a shared expert with a gate of its own), or absent.  Tensors are named embed, l<i>.norm1|norm2 (with .b and
.alpha), l<i>.mix.<name>, l<i>.mlp.<name> (l<i>.mlp.e<j>.<name>, l<i>.mlp.shared.<name>), final.norm, head.

A layer with `weights_of: j` is layer j run again: an `ExecStep` that names layer j's block and a cache plane (or state) of its own.
Planes are numbered like the layers of the configuration.
"""
from __future__ import annotations

from ..config.model_config import NesezenConfig
from ..parts.base import PartSpec
from .plan import ExecStep, ModelPlan

NO_POSITION_LIMIT = 1 << 30     # angles are computed from the position: nothing but int32 bounds it

_GATED = ("gate", "up", "down")


def _mixer(layer, D: int, eps: float, p: str, positions: dict) -> PartSpec:
    m = layer.mixer
    sizes = dict(hidden_size=D, num_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), eps=eps, prefix=p)
    if layer.type == "mlstm":
        return PartSpec("mlstm", dict(sizes, gate_cap=float(m["gate_cap"])))
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", dict(sizes, rot_dim=0, q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]),
                                                 scale=float(m["scale"]), window=None, position=None, gate="head"))
    rot, position = m.get("rot") or {}, None
    if int(rot.get("dims") or 0) > 0:
        position = p + "rot"
        positions[position] = PartSpec("rope", dict(head_dim=int(m["dim"]), rotary_dim=int(rot["dims"]), max_position=NO_POSITION_LIMIT,
                                                    theta=float(rot["base"]), interleaved=False, scaling=rot.get("scaling"),
                                                    table=False, precise=True))
    return PartSpec("attention_normed", dict(sizes, num_kv_heads=int(m["kv_heads"]), scale=float(m["scale"]),
                                             window=int((m.get("mask") or {}).get("size") or 0), position=position, bias=False,
                                             qk_norm=False, value_norm=False, sink=False, gate=False,
                                             softcap=float(m.get("softcap") or 0.0)))


def _feed_forward(mlp, D: int, p: str):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(hidden_size=D, intermediate_size=int(mlp["ff"]), prefix=p, names=_GATED))
    r, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", dict(
        hidden_size=D, expert_size=int(mlp["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), prefix=p,
        activation="silu_gated", scores="sigmoid", correction=False, weight_input=True, shared_gate="shared.sg",
        shared=dict(intermediate_size=int(shared["ff"]), prefix=p + "shared.", names=_GATED) if shared else None))


def nesezen_plan(cfg: NesezenConfig) -> ModelPlan:
    D = cfg.width
    norm = lambda name: PartSpec("tanh_stream", dict(size=D, weight_name=name))
    layers, positions, block_of, order = [], {}, {}, []
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is None:
            p = f"l{i}."
            ff = _feed_forward(layer.mlp, D, p + "mlp.")
            block_of[i] = len(layers)
            layers.append(PartSpec("pre_norm_stream", dict(
                mixer=_mixer(layer, D, cfg.eps, p + "mix.", positions), feed_forward=ff, input_norm=norm(p + "norm1"),
                post_mixer_norm=norm(p + "norm2") if ff else None, size=D)))
    for i in range(len(cfg.layers)):
        order.append(ExecStep(block_of[cfg.owner(i)], i, True))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_position=NO_POSITION_LIMIT,
        embedding_name="embed", lm_head_name="head", final_norm=norm("final.norm"), positions=positions, layers=layers, order=order,
        eos_token_id=None, default_dtype=cfg.torch_dtype)
