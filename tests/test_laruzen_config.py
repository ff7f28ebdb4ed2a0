"""Laruzen without a GPU: configuration, plan, tensor names, where per-request state lies, and closed forms of the plain
mechanisms (tests/plain/laruzen_plain.py)."""
import math

import pytest
import torch

from plain import laruzen_plain as P
from vllm_oxide_b200.cache.paged_cache import PagedCache
from vllm_oxide_b200.config import ConfigError, LaruzenConfig
from vllm_oxide_b200.models import CausalLM, resolve

YARN = {"factor": 3.0, "original": 96, "fast": 12.0, "slow": 2.0}


def gla(heads=3, dim=24, vdim=20, tau=9.0, **more):
    return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=tau, **more)}


def lightning(decay=(0.5, 0.75, 0.99), dim=12, vdim=28):
    return {"type": "lightning", "mixer": dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay))}


def sides(**more):
    left = dict(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.25, mask={"size": 21}, rot={"dims": 16, "base": 5000.0, "scaling": YARN})
    right = dict(width=36, blocks=3, conv=5)
    left.update({k[5:]: v for k, v in more.items() if k.startswith("left_")})
    right.update({k[6:]: v for k, v in more.items() if k.startswith("right_")})
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def config(layers, **more):
    return dict({"architecture": "Laruzen", "vocab": 90, "width": 48, "norm": {"eps": 1e-5},
                 "embedding": {"bigram": {"buckets": 31, "mul_prev": 7, "mul_cur": 3}}, "layers": layers}, **more)


MOE = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 28}}
DENSE = {"kind": "dense", "ff": 64}


def test_the_plan_follows_the_configuration():
    layers = [dict(gla(), mlp=DENSE), dict(sides(), mlp=MOE), dict(lightning(), mlp=None), dict(sides(left_rot=None, left_mask=None), mlp=DENSE)]
    cfg, plan = resolve(config(layers))
    assert isinstance(cfg, LaruzenConfig) and cfg.bigram == (31, 7, 3)
    assert [(s.layer, s.plane) for s in plan.order] == [(i, i) for i in range(4)]
    assert [l.kind for l in plan.layers] == ["sandwich"] * 4 and [l.params["shift"] for l in plan.layers] == [f"l{i}.shift" for i in range(4)]
    n = plan.layers[0].params
    assert all(n[k].params["one_plus"] for k in ("pre_mixer_norm", "post_mixer_norm", "pre_ff_norm", "post_ff_norm"))
    assert plan.final_norm.params["one_plus"] and plan.layers[2].params["pre_ff_norm"] is None
    a, b, c, d = (l.params["mixer"] for l in plan.layers)
    assert a.kind == "gated_linear_attention" and (a.params["tau"], a.params["rank"]) == (9.0, -1)
    assert c.kind == "lightning_attention" and c.params["decay"] == [0.5, 0.75, 0.99]
    assert b.kind == "side_by_side" and b.params["left"].kind == "attention_normed" and b.params["right"].kind == "recurrent_block"
    assert (b.params["left"].params["window"], b.params["left"].params["position"]) == (21, "l1.mix.left.rot")
    assert (d.params["left"].params["window"], d.params["left"].params["position"]) == (0, None) and list(plan.positions) == ["l1.mix.left.rot"]
    rope = plan.positions["l1.mix.left.rot"].params
    assert (rope["rotary_dim"], rope["head_dim"], rope["interleaved"], rope["table"], rope["scaling"]) == (16, 24, False, False, YARN)
    ff = plan.layers[1].params["feed_forward"]
    assert ff.kind == "routed_experts" and ff.params["shared"]["intermediate_size"] == 28
    assert (ff.params["activation"], ff.params["scores"], ff.params["normalise"], ff.params["correction"]) == ("silu_gated", "softmax", True, False)
    assert plan.layers[0].params["feed_forward"].kind == "swiglu" and plan.layers[0].params["feed_forward"].params["activation"] == "gelu_tanh"
    model = CausalLM(plan, torch.bfloat16, "cpu")
    names = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert names["embed"] == (90, 48) and names["bigram"] == (32, 48) and names["head"] == (90, 48) and names["final.norm"] == (48,)
    assert names["l0.mix.q"] == (72, 48) and names["l0.mix.v"] == (60, 48) and names["l0.mix.o"] == (48, 60) and names["l0.mix.norm"] == (20,)
    assert names["l0.mix.a1"] == (-1, 48) and names["l0.mix.a2"] == (72, -1) and names["l0.mix.a2.b"] == (72,) and names["l0.shift"] == (48,)
    assert names["l2.mix.norm"] == (84,) and names["l2.mix.g"] == (84, 48) and "l2.mlp.gate" not in names and "l2.norm2" not in names
    assert names["l1.mix.left.q"] == (96, 48) and names["l1.mix.left.v.b"] == (80,) and names["l1.mix.left.o.b"] == (48,)
    assert names["l1.mix.left.sink"] == (4,) and names["l1.mix.left.k.norm"] == (24,) and names["l1.mix.left.g"] == (160, 48)
    assert names["l1.mix.right.conv"] == (36, 5) and names["l1.mix.right.ra"] == (3, 12, 12) and names["l1.mix.right.ri.b"] == (3, 12)
    assert names["l1.mix.right.lam"] == (36,) and names["l1.mix.right.out"] == (48,) and names["l1.mix.left.out"] == (48,)
    assert names["l1.mlp.e5.down"] == (48, 20) and names["l1.mlp.shared.up"] == (28, 48) and names["l1.mlp.router"] == (6, 48)
    assert LaruzenConfig.from_dict(cfg.to_dict()) == cfg


def test_where_per_request_state_lies():
    """The mixer's floats, then the last normed row of the token shift; behind the planes, the token before, as an integer."""
    cfg, plan = resolve(config([dict(gla(), mlp=DENSE), dict(sides(), mlp=None), dict(lightning(), mlp=None)]))
    model = CausalLM(plan, torch.float32, "cpu")
    states, planes = model.state_specs(), model.cache_specs()
    assert [s.shape for s in states] == [(3 * 24 * 20 + 48,), (36 * 5 + 48,), (3 * 12 * 28 + 48,), (1,)]
    assert [s.dtype for s in states] == [torch.float32] * 3 + [torch.int32]
    assert [p is None for p in planes] == [True, False, True, True]
    assert (planes[1].kv_heads, planes[1].head_dim, planes[1].value_shape(), planes[1].window) == (2, 24, (2, 40), 21)
    cache = PagedCache(planes, states, torch.float32, "cpu", 16, 8, 2)
    assert cache.states[3].dtype == torch.int32 and cache.has_states
    cache.states[3].fill_(7)
    cache.states[0].fill_(1.5)
    cache.zero_states([1])
    assert cache.states[3].flatten().tolist() == [7, 0] and float(cache.states[0][1].abs().sum()) == 0.0 and float(cache.states[0][0, 0]) == 1.5
    # heads of two sizes are padded to one that the tensor-core kernels take, in 16 bits only
    assert CausalLM(plan, torch.bfloat16, "cpu").cache_specs()[1].head_dim == 48
    # a model without paged layers, one without a pair table
    cfg, plan = resolve(config([dict(gla(), mlp=None)], embedding={}))
    model = CausalLM(plan, torch.float32, "cpu")
    assert cfg.bigram is None and model.state_specs()[1] is None and "bigram" not in {s.name for s in model.tensor_specs()}
    assert LaruzenConfig.from_dict(cfg.to_dict()) == cfg


def test_stated_sizes_make_a_random_model_and_unstated_ones_cannot_be_drawn(tmp_path):
    from vllm_oxide_b200.engine.loading import write_random_model_folder
    with pytest.raises(ValueError, match="read from a checkpoint"):
        write_random_model_folder(str(tmp_path / "a"), config([dict(gla(), mlp=None)]), 1)
    write_random_model_folder(str(tmp_path / "b"), config([dict(gla(rank=5), mlp=MOE), dict(sides(), mlp=DENSE), dict(lightning(), mlp=None)]), 1)
    cfg, w = P.read_folder(str(tmp_path / "b"))
    assert w["l0.mix.a1"].shape == (5, 48) and P.forward(cfg, w, [1, 2, 3, 4, 5]).shape == (5, 90)


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][0]["mixer"].pop("tau"),
    lambda c: c["layers"][0]["mixer"].update(tau=0.0),
    lambda c: c["layers"][2]["mixer"]["decay"].pop(),
    lambda c: c["layers"][2]["mixer"].update(decay="slow"),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0),
    lambda c: c["layers"][1]["mixer"]["left"].update(heads=5),
    lambda c: c["layers"][1]["mixer"]["left"].pop("scale"),
    lambda c: c["layers"][1]["mixer"]["right"].update(blocks=5),
    lambda c: c["layers"][1]["mixer"].pop("right"),
    lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
    lambda c: c["embedding"]["bigram"].pop("buckets"),
    lambda c: c.pop("norm"),
])
def test_what_cannot_be_is_an_error(bad):
    import copy
    c = copy.deepcopy(config([dict(gla(), mlp=DENSE), dict(sides(), mlp=MOE), dict(lightning(), mlp=None)]))
    resolve(c)
    bad(c)
    with pytest.raises(ConfigError):
        resolve(c)


def test_plain_embedding_and_shift_in_closed_form():
    dt = torch.float64
    # rows of the pair table: the last one for the first token, else the hashed pair
    assert P.bigram_rows([4, 2, 9, 2], 7, 3, 31) == [31, (4 * 7 + 2 * 3) % 31, (2 * 7 + 9 * 3) % 31, (9 * 7 + 2 * 3) % 31]
    W = {"embed": torch.arange(20, dtype=dt).reshape(10, 2), "bigram": 100.0 * torch.arange(64, dtype=dt).reshape(32, 2)}
    x = P.embedded({"embedding": {"bigram": {"buckets": 31, "mul_prev": 7, "mul_cur": 3}}}, W, [4, 2], dt)
    assert x.tolist() == [[8.0 + 6200.0, 9.0 + 6300.0], [4.0 + 600.0, 5.0 + 700.0]]
    h = torch.tensor([[2.0, 4.0], [6.0, 0.0], [1.0, 1.0]], dtype=dt)
    assert P.token_shift(h, torch.tensor([0.5, 0.25], dtype=dt)).tolist() == [[1.0, 3.0], [4.0, 1.0], [3.5, 0.75]]


def test_plain_recurrences_in_closed_form():
    dt = torch.float64
    one = lambda *v: torch.tensor(v, dtype=dt)
    # one head, one key channel: S_t = f S + k v, o = S q, so o_t = q_t sum_s f^(t-s) k_s v_s
    q, k, v = one(1.0, 2.0, 3.0).reshape(3, 1, 1), one(1.0, -1.0, 2.0).reshape(3, 1, 1), one(4.0, 5.0, 6.0).reshape(3, 1, 1)
    o = P.matrix_recurrence(q, k, v, torch.full((3, 1, 1), 0.5, dtype=dt)).flatten().tolist()
    assert o == [4.0, 2.0 * (2.0 - 5.0), 3.0 * (0.5 * -3.0 + 12.0)]
    # the decay acts on the rows that belong to key channels
    q, k = one(1.0, 0.0, 1.0, 0.0).reshape(2, 1, 2), one(1.0, 1.0, 0.0, 0.0).reshape(2, 1, 2)
    decay = one(1.0, 1.0, 0.25, 0.75).reshape(2, 1, 2)
    assert P.matrix_recurrence(q, k, one(8.0, 9.0).reshape(2, 1, 1), decay).flatten().tolist() == [8.0, 2.0]
    # the channel recurrence with gates at one half: a = exp(-4 softplus(lam))
    W = {"r.ra": torch.zeros(1, 1, 1, dtype=dt), "r.ra.b": torch.zeros(1, 1, dtype=dt), "r.ri": torch.zeros(1, 1, 1, dtype=dt),
         "r.ri.b": torch.zeros(1, 1, dtype=dt), "r.lam": one(0.3)}
    a = math.exp(-4.0 * math.log1p(math.exp(0.3)))
    s = P.linear_recurrence(one(2.0, 3.0).reshape(2, 1), W, "r.", {"blocks": 1}, dt).flatten()
    first = math.sqrt(1 - a * a) * 0.5 * 2.0                         # also the first token's share is scaled by sqrt(1 - a^2)
    assert s.tolist() == pytest.approx([first, a * first + math.sqrt(1 - a * a) * 0.5 * 3.0])
    conv = P.causal_conv(one(1.0, 2.0, 4.0).reshape(3, 1), one(100.0, 10.0, 1.0).reshape(1, 3), one(0.5))
    assert conv[:, 0].tolist() == [1.5, 12.5, 124.5]
    assert P.gelu_tanh(one(0.0, 1.0)).tolist() == pytest.approx([0.0, 0.841192], abs=1e-6)


def test_plain_attention_in_closed_form():
    """One head of two dimensions, no rotation: the weights are exp(s) / (exp(sink) + sum exp(s)) over the window's keys."""
    dt = torch.float64
    eye, z2 = torch.eye(2, dtype=dt), torch.zeros(2, dtype=dt)
    W = {"a." + k: v for k, v in {"q": eye, "q.b": z2, "k": eye, "k.b": z2, "v": eye, "v.b": z2, "q.norm": torch.ones(2, dtype=dt),
                                  "k.norm": 2.0 * torch.ones(2, dtype=dt), "sink": torch.tensor([0.7], dtype=dt),
                                  "g": torch.zeros(2, 2, dtype=dt), "o": eye, "o.b": torch.tensor([10.0, 20.0], dtype=dt)}.items()}
    h = torch.tensor([[3.0, 0.0], [0.0, 5.0], [0.0, 1.0]], dtype=dt)
    m = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=0.25, mask={"size": 2})
    out = P.window_attention(h, W, "a.", m, 0.0, dt)
    r2 = math.sqrt(2.0)
    hit = math.exp(0.25 * r2 * 2.0 * r2)                             # a key along the query: (sqrt 2) * (2 sqrt 2) * scale
    sink = math.exp(0.7)
    # token 1 sees keys 0 (score 0) and 1; the gate is one half; values are unit in the root-mean-square sense
    assert out[1].tolist() == pytest.approx([10.0 + 0.5 * r2 / (1 + hit + sink), 20.0 + 0.5 * r2 * hit / (1 + hit + sink)])
    # token 2 no longer sees key 0
    assert out[2].tolist() == pytest.approx([10.0, 20.0 + 0.5 * r2 * 2 * hit / (2 * hit + sink)])
    # the softmax over the chosen logits alone
    idx, w, margin = P.route(torch.tensor([[3.0, 1.0, 2.0, 0.0]], dtype=dt), {"r.router": torch.eye(4, dtype=dt)}, "r.", 2, dt)
    assert idx.tolist() == [[0, 2]] and w[0].tolist() == pytest.approx([math.e / (1 + math.e), 1 / (1 + math.e)]) and margin.tolist() == [1.0]
