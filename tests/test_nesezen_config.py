"""Nesezen without a GPU: configuration, plan, tensor names, where per-request state lies, layers that use another layer's
tensors, and closed forms of the plain mechanisms (tests/plain/nesezen_plain.py)."""
import copy
import math

import pytest
import torch

from plain import nesezen_plain as P
from vllm_oxide_b200.cache.paged_cache import PagedCache
from vllm_oxide_b200.config import ConfigError, NesezenConfig
from vllm_oxide_b200.models import CausalLM, resolve

BY_WAVE = {"factor": 3.0, "original": 96, "low": 1.5, "high": 6.0}


def attention(**more):
    return {"type": "attention", "mixer": dict(dict(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.25, softcap=7.0, mask={"size": 21},
                                                    rot={"dims": 16, "base": 5000.0, "scaling": BY_WAVE}), **more)}


def mlstm(heads=3, dim=20, vdim=28, gate_cap=9.0):
    return {"type": "mlstm", "mixer": dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap)}


def latent(heads=5, dim=12, vdim=20, q_rank=30, kv_rank=36, scale=0.3):
    return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)}


def config(layers, **more):
    return dict({"architecture": "Nesezen", "vocab": 90, "width": 44, "norm": {"eps": 1e-4}, "layers": layers}, **more)


MOE = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 28}}
DENSE = {"kind": "dense", "ff": 64}


def test_the_plan_follows_the_configuration():
    layers = [dict(attention(), mlp=DENSE), dict(mlstm(), mlp=MOE), dict(latent(), mlp=None), dict(attention(rot=None, mask=None, softcap=None), mlp=DENSE)]
    cfg, plan = resolve(config(layers))
    assert isinstance(cfg, NesezenConfig) and [(s.layer, s.plane) for s in plan.order] == [(i, i) for i in range(4)]
    assert [l.kind for l in plan.layers] == ["pre_norm_stream"] * 4 and plan.final_norm.kind == "tanh_stream"
    assert plan.layers[2].params["post_mixer_norm"] is None and plan.layers[2].params["feed_forward"] is None
    a, b, c, d = (l.params["mixer"] for l in plan.layers)
    assert a.kind == "attention_normed" and (a.params["softcap"], a.params["window"], a.params["position"]) == (7.0, 21, "l0.mix.rot")
    assert not any(a.params[k] for k in ("bias", "qk_norm", "value_norm", "sink", "gate"))
    assert (d.params["softcap"], d.params["window"], d.params["position"]) == (0.0, 0, None) and list(plan.positions) == ["l0.mix.rot"]
    rope = plan.positions["l0.mix.rot"].params
    assert (rope["rotary_dim"], rope["head_dim"], rope["interleaved"], rope["table"], rope["scaling"]) == (16, 24, False, False, BY_WAVE)
    assert b.kind == "mlstm" and (b.params["gate_cap"], b.params["eps"]) == (9.0, 1e-4)
    assert c.kind == "latent_attention" and (c.params["rot_dim"], c.params["position"], c.params["gate"], c.params["window"]) == (0, None, "head", None)
    ff = plan.layers[1].params["feed_forward"]
    assert ff.kind == "routed_experts" and (ff.params["activation"], ff.params["scores"], ff.params["weight_input"]) == ("silu_gated", "sigmoid", True)
    assert ff.params["shared"]["intermediate_size"] == 28 and not ff.params.get("normalise")
    model = CausalLM(plan, torch.bfloat16, "cpu")
    names = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert names["embed"] == (90, 44) and names["head"] == (90, 44) and names["final.norm.alpha"] == () and names["final.norm.b"] == (44,)
    assert names["l0.norm1"] == (44,) and names["l0.norm2.alpha"] == () and "l2.norm2" not in names and "l2.norm2.b" not in names
    assert {n for n in names if n.startswith("l0.mix.")} == {"l0.mix." + k for k in "qkvo"} and names["l0.mix.v"] == (80, 44)
    assert {n[7:] for n in names if n.startswith("l1.mix.")} == {"q", "k", "v", "g", "o", "i", "i.b", "f", "f.b", "norm"}
    assert names["l1.mix.norm"] == (84,) and names["l1.mix.i"] == (3, 44) and names["l1.mix.f.b"] == (3,)
    assert names["l2.mix.g"] == (5, 44) and names["l2.mix.dkv"] == (36, 44) and names["l2.mix.uv"] == (100, 36) and names["l2.mix.dq.norm"] == (30,)
    assert names["l1.mlp.e5.down"] == (44, 20) and names["l1.mlp.shared.up"] == (28, 44) and names["l1.mlp.shared.sg"] == (1, 44)
    assert NesezenConfig.from_dict(cfg.to_dict()) == cfg
    # without a shared expert there is no gate of one either
    _, plan = resolve(config([dict(mlstm(), mlp={k: v for k, v in MOE.items() if k != "shared"})]))
    assert not [s.name for s in CausalLM(plan, torch.float32, "cpu").tensor_specs() if "shared" in s.name]


def test_where_per_request_state_and_pages_lie():
    cfg, plan = resolve(config([dict(mlstm(), mlp=DENSE), dict(attention(), mlp=None), dict(latent(), mlp=None)]))
    model = CausalLM(plan, torch.float32, "cpu")
    states, planes = model.state_specs(), model.cache_specs()
    # matrices, normalisers, maxima: 3 * (20 * 28 + 20 + 1), in whole groups of four floats
    assert states[0].shape == (1744,) and states[0].dtype == torch.float32 and states[1:] == [None, None]
    assert planes[0] is None and (planes[1].kv_heads, planes[1].head_dim, planes[1].value_shape(), planes[1].window) == (2, 24, (2, 40), 21)
    assert (planes[2].kv_heads, planes[2].head_dim, planes[2].tensors, planes[2].window) == (1, 48, 1, 0)      # a latent of 36, padded
    # heads of two sizes are padded to one that the tensor-core kernels take, in 16 bits only
    assert CausalLM(plan, torch.bfloat16, "cpu").cache_specs()[1].head_dim == 48
    cache = PagedCache(planes, states, torch.float32, "cpu", 16, 8, 2)
    cache.states[0].fill_(1.5)
    cache.zero_states([1])
    assert float(cache.states[0][1].abs().sum()) == 0.0 and float(cache.states[0][0, 0]) == 1.5


def test_a_layer_that_uses_another_layers_tensors():
    one, two = dict(attention(), mlp=MOE), dict(mlstm(), mlp=DENSE)
    cfg, plan = resolve(config([one, two, dict(one, weights_of=0), dict(two, weights_of=1), dict(one, weights_of=2), dict(latent(), mlp=None)]))
    assert [(s.layer, s.plane, s.write_cache) for s in plan.order] == [(0, 0, True), (1, 1, True), (0, 2, True), (1, 3, True), (0, 4, True), (2, 5, True)]
    assert len(plan.layers) == 3 and cfg.owner(4) == 0 and cfg.owner(5) == 5
    model = CausalLM(plan, torch.float32, "cpu")
    assert {s.name.split(".")[0] for s in model.tensor_specs() if s.name[0] == "l"} == {"l0", "l1", "l5"}
    # a cache and a state of its own for every run
    assert [p is not None for p in model.cache_specs()] == [True, False, True, False, True, True]
    assert [s is not None for s in model.state_specs()] == [False, True, False, True, False, False]
    assert NesezenConfig.from_dict(cfg.to_dict()) == cfg
    # a layer may use the tensors of one that comes later
    _, plan = resolve(config([dict(one, weights_of=1), one]))
    assert [(s.layer, s.plane) for s in plan.order] == [(0, 0), (0, 1)] and plan.layers[0].params["input_norm"].params["weight_name"] == "l1.norm1"


def test_a_random_folder_of_every_kind(tmp_path):
    from vllm_oxide_b200.engine.loading import write_random_model_folder
    one = dict(attention(), mlp=MOE)
    write_random_model_folder(str(tmp_path), config([one, dict(mlstm(), mlp=DENSE), dict(latent(), mlp=MOE), dict(one, weights_of=0)]), 1)
    cfg, w = P.read_folder(str(tmp_path))
    assert P.forward(cfg, w, [1, 2, 3, 4, 5]).shape == (5, 90) and float(w["l1.mix.f.b"].float().mean()) > 2.0


@pytest.mark.parametrize("bad", [
    lambda c: c["layers"][0].update(type="gla"),
    lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"].update(heads=5),
    lambda c: c["layers"][0]["mixer"].update(softcap=-1.0),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26),
    lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0),
    lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(low=6.0),
    lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("high"),
    lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0),
    lambda c: c["layers"][1]["mixer"].pop("vdim"),
    lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][2]["mixer"].pop("kv_rank"),
    lambda c: c["layers"][3].update(weights_of=3),
    lambda c: c["layers"][3].update(weights_of=4),
    lambda c: c["layers"][3].update(weights_of=1),
    lambda c: (c["layers"][3].update(weights_of=0), c["layers"][0].update(weights_of=3)),
    lambda c: c.pop("norm"),
])
def test_what_cannot_be_is_an_error(bad):
    c = copy.deepcopy(config([dict(attention(), mlp=DENSE), dict(mlstm(), mlp=MOE), dict(latent(), mlp=None), dict(attention(), mlp=DENSE, weights_of=0)]))
    resolve(c)
    bad(c)
    with pytest.raises(ConfigError):
        resolve(c)


def test_frequencies_stretched_by_wavelength():
    """The package's frequencies against the rule spelled out, with waves on either side of both borders and between them; an
    angle of zero scaling is the plain one."""
    from vllm_oxide_b200.parts.rope import scaled_frequencies
    for dims, base, s in ((64, 1e4, BY_WAVE), (16, 50.0, BY_WAVE), (32, 500000.0, {"factor": 8.0, "original": 8192, "low": 1.0, "high": 4.0})):
        want = P.stretched_frequencies(dims, base, s)
        plain = P.stretched_frequencies(dims, base, None)
        got, amplitude = scaled_frequencies(dims, base, s, precise=True)
        assert amplitude == 1.0 and torch.allclose(got.double(), want, rtol=1e-6)
        ratio = plain / want
        assert ratio.min() == pytest.approx(1.0) and ratio.max() == pytest.approx(s["factor"]) and bool(((ratio > 1.01) & (ratio < s["factor"] - 0.01)).any())
    # wave 60 of a length of 96: turns 1.6, a share of 0.1 / 4.5
    f = 2 * math.pi / 60.0
    got, _ = scaled_frequencies(2, 1.0, {"factor": 3.0, "original": 96 * f, "low": 1.5, "high": 6.0}, precise=True)    # one pair, f = 1
    share = (96 * f / (2 * math.pi) - 1.5) / 4.5
    assert float(got[0]) == pytest.approx((1 - share) / 3.0 + share)
    with pytest.raises(ValueError, match="low"):
        scaled_frequencies(8, 1e4, {"factor": 2.0, "original": 10, "low": 4.0, "high": 4.0})


def test_plain_norm_and_feed_forwards_in_closed_form():
    dt = torch.float64
    one = lambda *v: torch.tensor(v, dtype=dt)
    assert P.tanh_norm(one(0.0, 2.0), 0.5, one(3.0, 4.0), one(1.0, -1.0)).tolist() == pytest.approx([1.0, 4.0 * math.tanh(1.0) - 1.0])
    # one expert of one feature, two experts, one chosen: its weight enters twice, once in the gate and once in the up value
    silu = lambda z: z / (1 + math.exp(-z))
    W = {"f.router": one(1.0, -1.0).reshape(2, 1), "f.shared.sg": one(0.5).reshape(1, 1)}
    for name, g, u, d in (("e0", 2.0, 3.0, 5.0), ("e1", 1.0, 1.0, 1.0), ("shared", 1.0, 2.0, 4.0)):
        W.update({f"f.{name}.gate": one(g).reshape(1, 1), f"f.{name}.up": one(u).reshape(1, 1), f"f.{name}.down": one(d).reshape(1, 1)})
    h, s = 0.7, 1 / (1 + math.exp(-0.7))
    mlp = {"router": {"experts": 2, "top": 1}, "shared": {"ff": 1}}
    want = 5.0 * silu(2.0 * s * h) * 3.0 * s * h + 4.0 * silu(h) * 2.0 * h / (1 + math.exp(-0.5 * h))
    assert P.moe_ff(one(h).reshape(1, 1), W, "f.", mlp, dt).item() == pytest.approx(want)


def test_plain_exponential_gates_in_closed_form():
    """One head, one key and value channel: against the sums written out without a running maximum, S = sum_s w_s k_s v_s,
    n = sum_s w_s k_s with w_s = exp(i_s + f_{s+1} + ... + f_t), o = S q / max(|n q|, 1) where exp(-m) scales to 1."""
    dt = torch.float64
    g = torch.Generator().manual_seed(4)
    n = 9
    q, k, v = (torch.randn(n, 1, 1, generator=g, dtype=dt) for _ in range(3))
    i, f = P.mlstm_gates(3.0 * torch.randn(n, 1, generator=g, dtype=dt), torch.randn(n, 1, generator=g, dtype=dt), 4.0)
    assert float(i.abs().max()) < 4.0 and float(f.max()) < 0.0
    o = P.mlstm_recurrence(q, k, v, i, f).flatten()
    m = 0.0
    for t in range(n):
        m = max(float(f[t]) + m, float(i[t]))
        w = [math.exp(float(i[s]) + float(f[s + 1:t + 1].sum())) for s in range(t + 1)]
        S = sum(w[s] * float(k[s]) * float(v[s]) for s in range(t + 1)) * float(q[t])
        z = sum(w[s] * float(k[s]) for s in range(t + 1)) * float(q[t])
        # the same, scaled by exp(-m): the floor of the normaliser is then 1, what is added to it 1e-6 exp(m)
        assert float(o[t]) == pytest.approx(S / (max(abs(z), 1.0) + 1e-6 * math.exp(m)), rel=1e-9)
    assert P.log_sigmoid(torch.tensor([0.0, -40.0, 40.0], dtype=dt)).tolist() == pytest.approx([-math.log(2.0), -40.0, -math.exp(-40.0)])


def test_plain_attention_in_closed_form():
    """One head of two dimensions, no rotation: the scores are capped before the softmax, and a key behind the window is not
    there."""
    dt = torch.float64
    eye = torch.eye(2, dtype=dt)
    W = {"a." + k: eye for k in "qkvo"}
    h = torch.tensor([[3.0, 0.0], [0.0, 5.0], [0.0, 1.0]], dtype=dt)
    m = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=0.5, softcap=2.0, mask={"size": 2})
    out = P.attention(h, W, "a.", m, 0.0, dt)
    hit = math.exp(2.0 * math.tanh(12.5 / 2.0))
    assert out[1].tolist() == pytest.approx([3.0 / (1 + hit), 5.0 * hit / (1 + hit)])
    a, b = math.exp(2.0 * math.tanh(2.5 / 2.0)), math.exp(2.0 * math.tanh(0.5 / 2.0))
    assert out[2].tolist() == pytest.approx([0.0, (5.0 * a + b) / (a + b)])
    # through a latent of one number: keys and values are multiples of it, a gate of one half for the one head
    one = lambda *v: torch.tensor(v, dtype=dt)
    W = {"m.dq": one(1.0, 0.0).reshape(1, 2), "m.dq.norm": one(2.0), "m.uq": one(1.0).reshape(1, 1), "m.dkv": one(0.0, 1.0).reshape(1, 2),
         "m.dkv.norm": one(3.0), "m.uk": one(1.0).reshape(1, 1), "m.uv": one(10.0).reshape(1, 1), "m.g": torch.zeros(1, 2, dtype=dt), "m.o": torch.ones(2, 1, dtype=dt)}
    out = P.latent_attention(torch.tensor([[4.0, 7.0], [-1.0, -5.0]], dtype=dt), W, "m.", dict(heads=1, dim=1, vdim=1, scale=0.1), 0.0, dt)
    assert out[0].tolist() == pytest.approx([15.0, 15.0])              # rms-normed to 1: a latent of 3, a value of 30
    e = math.exp(0.1 * -2.0 * -3.0) / (math.exp(0.1 * -2.0 * -3.0) + math.exp(0.1 * -2.0 * 3.0))
    assert out[1, 0].item() == pytest.approx(0.5 * (30.0 * (1 - e) - 30.0 * e))
