"""Every mechanism of Nesezen alone, as a part with pages and state slots of its own, against its plain function
(tests/plain/nesezen_plain.py): the stream's step with its norm, the matrix memory with exponential gates at every width of its scan
(whole, decoded, in portions, cut along the tokens), attention with capped scores on the plain and on the tensor-core kernels,
latent attention with a gate a head, experts weighted at their inputs beside a gated shared one on every path of their products."""
import pytest
import torch

from helpers import DEV, Alone, assert_close, held, make_context, rand
from plain import nesezen_plain as P

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


@pytest.fixture(scope="module", autouse=True)
def few_threads():
    """The plain functions are many small operations: a pool of threads only slows them down."""
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 4))
    yield
    torch.set_num_threads(n)


def load(part, w, dt):
    """Gives a part the tensors it lists, each in the type the engine keeps it in."""
    from vllm_oxide_b200.weights.loader import kept_dtype
    part.load({s.name: w[s.name].to(kept_dtype(s.role, dt)).to(DEV).contiguous() for s in part.tensor_specs()})


def draw(part, seed):
    """Random tensors for everything the part lists (float64): matrices by their fan-in, gains near one, the rest small."""
    w = {}
    for i, s in enumerate(part.tensor_specs()):
        shape = tuple(s.shape)
        if s.role == "matrix":
            w[s.name] = rand(shape, seed + i, shape[-1] ** -0.5)
        elif s.role == "norm":
            w[s.name] = 1.0 + 0.2 * rand(shape, seed + i)
        else:
            w[s.name] = rand(shape, seed + i, 0.4)
    return w


def hold(part, w, dt):
    """The same tensors as the plain functions should see them: what the engine keeps in float as it is, the rest rounded."""
    from vllm_oxide_b200.weights.loader import kept_dtype
    roles = {s.name: s.role for s in part.tensor_specs()}
    return {k: (v.float().double() if kept_dtype(roles[k], dt) == torch.float32 else held(v, dt)) for k, v in w.items()}


def run_cuts(part, x, cuts_list, want, dt, what, tol=None, slots=2, pages=40, kernels_ran=None):
    """Feeds x [n, D] in several cuts, each as a request of its own over pages and slots that the ones before used."""
    from vllm_oxide_b200 import kernels
    alone = Alone([part], dt, block_size=16, slots=slots, pages=pages)
    kernels.enable_kernel_timers(True)
    try:
        for k, cuts in enumerate(cuts_list):
            at, rows, i = 0, [], 0
            while at < x.shape[0]:
                n = min(cuts[i % len(cuts)], x.shape[0] - at)
                i += 1
                rows.append(alone.step([(100 + k, x[at:at + n])], end=[100 + k] if at + n == x.shape[0] else [])[0])
                at += n
            assert_close(torch.cat(rows), want, dt, f"{what}, cuts {cuts[:4]}", tol)
        if kernels_ran is not None:
            kernels_ran.update(kernels.kernel_timer_report())
    finally:
        kernels.enable_kernel_timers(False)


# ---------------------------------------------------------------- the stream's step with its norm
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D", [8, 30, 64, 516, 1040, 2052, 4100, 8195])
def test_the_elementwise_norm_around_the_stream(D, dt):
    from vllm_oxide_b200 import kernels
    n, f32 = 5, torch.float32
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = lambda t, d=dt: t.to(d).to(DEV).contiguous()
    x = rand((n, D), 1, 3.0).float().double()
    x[0, :6] = torch.tensor([0.0, 1e-6, -1e-6, 300.0, -300.0, 1e5], dtype=torch.float64)      # small, and far into both flat ends
    y, z = held(rand((n, D), 2), dt), held(rand((n, D), 6), dt)
    y[0, :6], z[0, :6] = 0.0, 0.0
    w, b, alpha = (1.0 + 0.3 * rand((D,), 3)).float().double(), rand((D,), 4, 0.3).float().double(), torch.tensor([0.7]).double()
    a = dev(alpha.float(), f32)
    norm = lambda t: P.tanh_norm(t, alpha.float().double(), w, b)
    stream, out = dev(x, f32), torch.empty((n, D), dtype=dt, device=DEV)
    kernels.tanh_norm_step(stream, err, y1=dev(y), alpha=a, w=dev(w, f32), b=dev(b, f32), out=out)
    assert_close(stream, x + y, f32, "stream", 1e-6)
    assert_close(out, norm(x + y), dt, "normed", 1e-6 if dt == f32 else 0.005)
    kernels.tanh_norm_step(stream, err, y1=dev(y), y2=dev(z))                                    # two outputs, no norm
    assert_close(stream, x + y + (y + z), f32, "two outputs", 1e-6)
    want, before = x + y + (y + z), stream.clone()
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
    some = torch.empty((3, D), dtype=dt, device=DEV)
    kernels.tanh_norm_step(stream, err, y1=dev(y), alpha=a, w=dev(w, f32), out=some, rows=rows, n_out=3)      # no bias
    assert torch.equal(stream, before) and int(err.item()) == 0
    assert_close(some, (norm(want + y) - b)[[4, 0, 4]], dt, "chosen rows", 2e-6 if dt == f32 else 0.005)
    kernels.tanh_norm_step(stream, err, y1=dev(y), alpha=a, w=dev(w, f32), b=dev(b, f32), out=out, init=True)
    assert_close(stream, y, f32, "a stream that begins", 1e-6)
    assert_close(out, norm(y), dt, "the first norm", 1e-6 if dt == f32 else 0.005)
    kernels.tanh_norm_step(stream, err, y1=dev(y), alpha=a, w=dev(w, f32), out=some, rows=torch.tensor([0, 5, -1], dtype=torch.int32, device=DEV), n_out=3)
    assert int(err.item()) == 16, "rows outside the batch are named, not read"


@pytest.mark.parametrize("norm", ["tanh_stream", "layernorm_stream", "rmsnorm_parallel_stream"])
def test_the_block_takes_any_norm_of_a_float_stream(norm):
    from vllm_oxide_b200.cache.paged_cache import PagedCache
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, n, dt = 24, 7, torch.float32
    common = dict(size=D) if norm == "tanh_stream" else dict(size=D, eps=EPS)
    spec = lambda name: PartSpec(norm, dict(common, weight_name=name))
    mixer = PartSpec("mlstm", dict(hidden_size=D, num_heads=2, dim=8, vdim=12, gate_cap=5.0, eps=EPS, prefix="m."))
    ff = PartSpec("swiglu", dict(hidden_size=D, intermediate_size=40, prefix="f.", names=("gate", "up", "down")))
    part = build_part("block", PartSpec("pre_norm_stream", dict(mixer=mixer, feed_forward=ff, input_norm=spec("n1"), post_mixer_norm=spec("n2"), size=D)),
                      positions={}, dtype=dt, device=DEV)
    w = draw(part, 3)
    load(part, w, dt)
    wh = hold(part, w, dt)
    plain = {"tanh_stream": lambda x, k: P.tanh_norm(x, wh.get(k + ".alpha"), wh[k], wh.get(k + ".b")),
             "layernorm_stream": lambda x, k: (x - x.mean(-1, keepdim=True)) / torch.sqrt(x.var(-1, unbiased=False, keepdim=True) + EPS) * wh[k],
             "rmsnorm_parallel_stream": lambda x, k: P.rms(x, EPS) * wh[k]}[norm]
    cache = PagedCache([None], [part.state_spec()], dt, DEV, 16, 4, 1)
    assert cache.manager.add_request(0) and cache.manager.ensure(0, 0, n)
    ctx = make_context(cache.manager, [(0, 0, [0] * n, [])], dt)
    cache.zero_states([0])
    x = rand((n, D), 9).float().double()
    hidden, stream = part.forward(x.float().to(DEV), None, ctx, None, cache.states[0])
    x = x + P.mlstm(plain(x, "n1"), wh, "m.", dict(heads=2, dim=8, vdim=12, gate_cap=5.0), EPS, torch.float64)
    assert_close(stream, x, dt, norm + ": stream")
    assert_close(hidden, P.gated_ff(plain(x, "n2"), wh, "f.", torch.float64), dt, norm + ": pending")
    with pytest.raises(ValueError, match="kind"):
        build_part("block", PartSpec("pre_norm_stream", dict(mixer=mixer, feed_forward=None, input_norm=PartSpec("rmsnorm", dict(size=D, eps=EPS, weight_name="n")),
                                                             post_mixer_norm=None, size=D)), positions={}, dtype=dt, device=DEV)


# ---------------------------------------------------------------- the matrix memory with exponential gates
# A head's norm makes a small sum of large terms as loud as any other, so in 16 bits the plain function is given the projections as
# the engine holds them: rounded.  What is left is the engine's own arithmetic.
def plain_memory(x, wh, m, dt):
    return P.mlstm(x, wh, "m.", m, EPS, torch.float64, noise=None if dt == torch.float32 else lambda t: held(t, dt))


SCANS = [(3, 16, 8), (2, 24, 20), (1, 32, 32), (5, 12, 40), (2, 64, 48), (3, 128, 12), (1, 200, 36), (2, 8, 3), (1, 1, 16), (2, 128, 128), (2, 48, 200),
         (1, 36, 600)]


def mlstm_part(dt, D, m):
    from vllm_oxide_b200.parts import PartSpec, build_part
    return build_part("mixer", PartSpec("mlstm", dict(hidden_size=D, num_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=m["gate_cap"], eps=EPS,
                                                      prefix="m.")), dtype=dt, device=DEV)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", SCANS)
def test_matrix_memory(heads, dim, vdim, dt):
    D, m = (64, 72, 40)[dim % 3], dict(heads=heads, dim=dim, vdim=vdim, gate_cap=6.0)
    part = mlstm_part(dt, D, m)
    w = draw(part, 11)
    # heads that forget at rates of their own, input gates up to their cap; normalisers that count and floors that count
    w["m.f.b"] = torch.linspace(-1.0, 5.0, heads, dtype=torch.float64) if heads > 1 else torch.tensor([3.0], dtype=torch.float64)
    w["m.i"] = 3.0 * w["m.i"]
    load(part, w, dt)
    x = held(rand((330, D), 5), dt)
    want = plain_memory(x, hold(part, w, dt), m, dt)
    run_cuts(part, x, [[330], [290] + [1] * 40, [7, 2, 33, 90], [2], [17, 16]], want, dt, f"mlstm {heads} x {dim} x {vdim}",
             5e-5 if dt == torch.float32 else 0.04)


def gates_and_normalisers(m, w, x):
    """The plain running maxima [n, H] and normaliser read-outs scaled by exp(m)."""
    n, H, dk = x.shape[0], m["heads"], m["dim"]
    q, k = (x @ w["m.q"].T).reshape(n, H, dk) * dk ** -0.5, (x @ w["m.k"].T).reshape(n, H, dk)
    i, f = P.mlstm_gates(x @ w["m.i"].T + w["m.i.b"], x @ w["m.f"].T + w["m.f.b"], m["gate_cap"])
    run, z, ms, nq = x.new_zeros(H), x.new_zeros((H, dk)), [], []
    for t in range(n):
        new = torch.maximum(f[t] + run, i[t])
        z = torch.exp(f[t] + run - new)[:, None] * z + torch.exp(i[t] - new)[:, None] * k[t]
        run = new
        ms.append(new)
        nq.append((z * q[t]).sum(-1).abs() * torch.exp(new))
    return torch.stack(ms), torch.stack(nq)


def test_the_floor_and_the_normaliser_both_decide():
    """Tokens whose normaliser lies below its floor and above it, and maxima that rise and fall, in one run; a maximum that
    started at minus infinity, or a normaliser that were left out, would show in the first rows."""
    D, m = 40, dict(heads=2, dim=24, vdim=20, gate_cap=8.0)
    dt = torch.float32
    part = mlstm_part(dt, D, m)
    w = draw(part, 21)
    w["m.i"], w["m.f.b"] = 4.0 * w["m.i"], torch.tensor([1.0, 4.0], dtype=torch.float64)
    w["m.i.b"] = torch.tensor([-5.0, 1.0], dtype=torch.float64)
    load(part, w, dt)
    x = held(rand((200, D), 7), dt)
    wh = hold(part, w, dt)
    ms, nq = gates_and_normalisers(m, wh, x)
    assert 0.1 < float((nq > 1.0).double().mean()) < 0.9 and float(ms.min()) < 0.0 < float(ms.max()), "both branches of the denominator"
    assert float(ms[0, 0]) > -1.5, "the maximum starts at zero: the first input gate lies far below it"
    want = P.mlstm(x, wh, "m.", m, EPS, torch.float64)
    run_cuts(part, x, [[200], [1], [2], [33, 1, 90]], want, dt, "floors", 5e-5)


@pytest.mark.parametrize("n", [700, 2500])
def test_a_memory_that_lasts(n):
    """With forget gates of all but one, the last rows hang on what the first tokens wrote, in every cut (2,500 tokens: several
    tokens a thread of the gates' scan, and the most ranges)."""
    D, m = 32, dict(heads=2, dim=48, vdim=24, gate_cap=12.0)
    dt = torch.float32
    part = mlstm_part(dt, D, m)
    w = draw(part, 3)
    w["m.f.b"] = w["m.f.b"] + 11.0
    w["m.i.b"] = torch.tensor([0.5, -2.0], dtype=torch.float64)
    load(part, w, dt)
    wh = hold(part, w, dt)
    x = held(rand((n, D), 7), dt)
    want = P.mlstm(x, wh, "m.", m, EPS, torch.float64)
    if n == 700:
        other = x.clone()
        other[:10] = rand((10, D), 8, 3.0)
        assert (P.mlstm(other, wh, "m.", m, EPS, torch.float64) - want)[-1].abs().max() > 0.02 * want[-1].abs().max()
    run_cuts(part, x, [[n], [n - 300] + [3] * 100, [n - 50] + [1] * 50], want, dt, "a lasting memory", 1e-4, pages=170)


def test_gates_at_the_ends_of_their_range():
    """Input gates that leap from floor to cap over a few tokens and forget gates that erase: factors of exp(-30), no overflow,
    no loss where the maximum falls again."""
    D, m = 24, dict(heads=3, dim=16, vdim=8, gate_cap=15.0)
    for dt in DTYPES:
        part = mlstm_part(dt, D, m)
        w = draw(part, 33)
        w["m.i"] = 12.0 * w["m.i"]
        w["m.f.b"] = torch.tensor([-14.0, 0.0, 6.0], dtype=torch.float64)
        load(part, w, dt)
        x = held(rand((150, D), 5), dt)
        wh = hold(part, w, dt)
        ms, _ = gates_and_normalisers(m, wh, x)
        assert float(ms.max()) > 12.0 and float(ms.min()) < -8.0
        want = plain_memory(x, wh, m, dt)
        run_cuts(part, x, [[150], [120] + [1] * 30, [2, 35]], want, dt, "extreme gates", 1e-4 if dt == torch.float32 else 0.06)


@pytest.mark.parametrize("dt", DTYPES)
def test_unequal_requests_over_slots_used_again(dt):
    D, m = 48, dict(heads=2, dim=24, vdim=16, gate_cap=7.0)
    part = mlstm_part(dt, D, m)
    w = draw(part, 31)
    w["m.f.b"] = w["m.f.b"] + 4.0
    load(part, w, dt)
    wh = hold(part, w, dt)
    alone = Alone([part], dt, block_size=16, pages=30, slots=2)
    xs = {rid: held(rand((n, D), 40 + rid), dt) for rid, n in ((1, 100), (2, 37), (3, 64), (4, 5), (5, 190))}
    got, at = {rid: [] for rid in xs}, {rid: 0 for rid in xs}
    for portions in [[(1, 50)], [(1, 1), (2, 30)], [(1, 49), (2, 7)], [(3, 64)], [(4, 5), (5, 2)], [(5, 188)]]:
        batch = [(rid, xs[rid][at[rid]:at[rid] + n]) for rid, n in portions]
        out = alone.step(batch, end=[rid for rid, n in portions if at[rid] + n == xs[rid].shape[0]])[0]
        k = 0
        for rid, rows in batch:
            got[rid].append(out[k:k + rows.shape[0]])
            at[rid] += rows.shape[0]
            k += rows.shape[0]
    assert alone.m.num_free_state_slots == 2
    for rid, x in xs.items():
        assert_close(torch.cat(got[rid]), plain_memory(x, wh, m, dt), dt, f"request {rid}", 5e-5 if dt == torch.float32 else 0.04)


@pytest.mark.parametrize("chunks", [1, 2, 3, 7, 16])
@pytest.mark.parametrize("dk, dv", [(24, 20), (128, 128), (64, 200)])
def test_ranges_of_a_portion_are_one_walk(chunks, dk, dv):
    """The scan cut into any number of ranges, from a state that is not zero, with a slot of its own for two requests: outputs,
    normalisers and what is left in the slots are those of the walk in one piece."""
    from vllm_oxide_b200 import kernels
    H, T, f32 = 2, 150, torch.float32
    off = 2 * H * dk + 2 * H * dv
    rows = rand((T, off + 2 * H), 3).float().to(DEV)
    bi, bf, nw = (rand((n,), s).float().to(DEV) for n, s in ((H, 4), (H, 5), (H * dv, 6)))
    bf += 3.0
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    cu = torch.tensor([0, 90, T], dtype=torch.int32, device=DEV)
    slots = torch.tensor([2, 0], dtype=torch.int32, device=DEV)
    start = rand((3, H * (dk * (dv + 1) + 1) + 5), 7).float().to(DEV)

    def run(c):
        state = start.clone()
        gates, raw, nq = (torch.empty((T, n), dtype=f32, device=DEV) for n in (H * 4, H * dv, H))
        scratch = torch.empty(2 * c * H * dk * (dv + 2), dtype=f32, device=DEV)
        kernels.mlstm_scan(rows, off, off + H, 2 * H * dk + H * dv, bi, bf, nw, state, cu, slots, 2, H, dk, dv, dk ** -0.5, 6.0, EPS, err, gates=gates,
                           raw=raw, nq=nq, chunks=c, scratch=scratch)
        return state, gates, raw, nq
    one, many = run(1), run(chunks)
    assert int(err.item()) == 0
    for a, b, what in zip(one, many, ("state", "gates", "outputs", "normalisers")):
        assert_close(b, a, f32, f"{what} in {chunks} ranges", 2e-5)
    assert torch.equal(many[0][1], start[1]) and torch.equal(many[0][:, -5:], start[:, -5:]), "a slot nobody uses, and what lies behind a row"


# ---------------------------------------------------------------- attention with capped scores
BY_WAVE = {"factor": 4.0, "original": 64, "low": 1.0, "high": 4.0}
ATTENTION = {
    # (D, sizes, fast in 16 bits): padded to 48, 64 and 128 (TMA, tcgen05), 32 (cp.async); more query heads than those kernels take
    "values wider than keys": (40, dict(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.5, softcap=4.0, mask={"size": 19}, rot={"dims": 16, "base": 100.0, "scaling": BY_WAVE}), True),
    "64 wide, the whole head turns": (64, dict(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.3, softcap=3.0, mask={"size": 44}, rot={"dims": 64, "base": 1e4, "scaling": BY_WAVE}), True),
    "128 wide, a window of one tile": (48, dict(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.2, softcap=2.0, mask={"size": 64}, rot={"dims": 32, "base": 1e4}), True),
    "keys wider than values": (32, dict(heads=3, kv_heads=3, dim=40, vdim=16, scale=0.5, softcap=5.0, mask={"size": 23}, rot={"dims": 10, "base": 777.0, "scaling": BY_WAVE}), True),
    "a window of one, one head": (32, dict(heads=1, kv_heads=1, dim=16, vdim=32, scale=0.3, softcap=1.0, mask={"size": 1}, rot={"dims": 16, "base": 50.0}), True),
    "no window, no rotation": (32, dict(heads=6, kv_heads=2, dim=16, vdim=16, scale=0.6, softcap=2.5, mask=None, rot=None), True),
    "no cap": (32, dict(heads=6, kv_heads=2, dim=32, vdim=32, scale=0.3, softcap=0.0, mask={"size": 30}, rot={"dims": 32, "base": 1e4}), True),
    "odd sizes": (32, dict(heads=2, kv_heads=1, dim=9, vdim=7, scale=0.8, softcap=3.0, mask={"size": 33}, rot={"dims": 6, "base": 60.0}), True),
    "twenty heads on one": (32, dict(heads=20, kv_heads=1, dim=16, vdim=16, scale=0.5, softcap=2.0, mask={"size": 50}, rot={"dims": 8, "base": 1e4}), False),
}


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", sorted(ATTENTION))
def test_windowed_attention_with_capped_scores(case, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, m, fast = ATTENTION[case]
    rot, positions, position = m.get("rot"), {}, None
    if rot:
        position = "r"
        positions["r"] = build_part("position", PartSpec("rope", dict(head_dim=m["dim"], rotary_dim=rot["dims"], max_position=1 << 30, theta=rot["base"],
                                                                      interleaved=False, table=False, precise=True, scaling=rot.get("scaling"))), device=DEV)
    part = build_part("mixer", PartSpec("attention_normed", dict(
        hidden_size=D, num_heads=m["heads"], num_kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], eps=EPS, prefix="m.",
        window=(m.get("mask") or {}).get("size"), position=position, bias=False, qk_norm=False, value_norm=False, sink=False, gate=False,
        softcap=m["softcap"])), positions=positions, dtype=dt, device=DEV)
    w = draw(part, 21)
    w["m.q"], w["m.k"] = 1.5 * w["m.q"], 1.5 * w["m.k"]
    load(part, w, dt)
    x = held(rand((200, D), 6), dt)
    wh = hold(part, w, dt)
    want = P.attention(x, wh, "m.", m, EPS, torch.float64)
    if m["softcap"] and (m.get("mask") or {}).get("size") != 1:
        assert (P.attention(x, wh, "m.", dict(m, softcap=0.0), EPS, torch.float64) - want).abs().max() > 0.05 * want.abs().max(), "the cap counts"
    ran = {}
    run_cuts(part, x, [[200], [150] + [1] * 50, [7, 2, 33, 64], [2]], want, dt, case, kernels_ran=ran)
    if dt == torch.bfloat16 and fast:
        assert "paged_attention_generic" not in ran and any(k.startswith("attention_prefill") for k in ran) and \
            any(k.startswith("attention_decode") for k in ran), ran
    else:
        assert "paged_attention_generic" in ran


# ---------------------------------------------------------------- latent attention
LATENT = {
    # (D, sizes, fast in 16 bits)
    "a latent of 64": (48, dict(heads=4, dim=16, vdim=24, q_rank=40, kv_rank=64, scale=0.4), True),
    "a latent that is padded": (40, dict(heads=3, dim=20, vdim=12, q_rank=17, kv_rank=37, scale=0.4), True),
    "one head, ranks of one": (32, dict(heads=1, dim=8, vdim=8, q_rank=1, kv_rank=1, scale=0.5), True),
    "more heads than a group": (64, dict(heads=21, dim=8, vdim=8, q_rank=32, kv_rank=48, scale=0.5), True),
    "a latent wider than the fast kernels": (64, dict(heads=2, dim=16, vdim=16, q_rank=64, kv_rank=272, scale=0.3), False),
    "values as wide as the latent": (64, dict(heads=8, dim=64, vdim=128, q_rank=128, kv_rank=128, scale=0.15), True),
}


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", sorted(LATENT))
def test_latent_attention_with_a_gate_a_head(case, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, m, fast = LATENT[case]
    part = build_part("mixer", PartSpec("latent_attention", dict(hidden_size=D, num_heads=m["heads"], dim=m["dim"], rot_dim=0, vdim=m["vdim"],
                                                                 q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=m["scale"], eps=EPS, window=None,
                                                                 position=None, prefix="m.", gate="head")), positions={}, dtype=dt, device=DEV)
    w = draw(part, 41)
    w["m.g"], w["m.uq"] = 3.0 * w["m.g"], 2.0 * w["m.uq"]
    load(part, w, dt)
    x = held(rand((200, D), 8), dt)
    wh = hold(part, w, dt)
    want = P.latent_attention(x, wh, "m.", m, EPS, torch.float64)
    assert (0.5 / P.sigmoid(x @ wh["m.g"].T)).std() > 0.3, "the gates differ"
    ran = {}
    run_cuts(part, x, [[200], [150] + [1] * 50, [7, 2, 33, 64], [2]], want, dt, case, 3e-5 if dt == torch.float32 else 0.04, kernels_ran=ran)
    assert ("paged_attention_generic" not in ran) == (dt == torch.bfloat16 and fast), ran


# ---------------------------------------------------------------- experts
def run_ff(part, x, dt):
    from vllm_oxide_b200.cache.paged_cache import PagedCache
    n = x.shape[0]
    cache = PagedCache([None], [None], dt, DEV, 16, 2 + n // 16, 1)
    assert cache.manager.add_request(0) and cache.manager.ensure(0, 0, n)
    ctx = make_context(cache.manager, [(0, 0, [0] * n, [])], dt)
    got = part.forward(x.to(dt).to(DEV).contiguous(), ctx)
    assert int(ctx.err.item()) == 0
    return got


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D, I, E, top, shared, n", [
    (64, 24, 12, 2, 40, 40),         # few pairs: the experts' rows are streamed pair by pair in bfloat16
    (48, 16, 6, 6, 8, 9),            # every expert chosen
    (40, 8, 5, 1, 24, 5),            # one expert: its weight is not one
    (128, 64, 8, 4, 64, 300),        # enough pairs for the tcgen05 products in bfloat16
    (160, 48, 9, 1, 96, 700),        # the same with one choice a token
    (72, 33, 4, 2, 17, 3),           # odd widths: the float-accumulating tile kernel
    (70, 12, 3, 2, 10, 400),         # the same with many tokens
    (64, 24, 1, 1, 40, 7),           # a single expert
    (64, 24, 7, 3, 0, 20),           # no shared expert
])
def test_experts_weighted_at_their_inputs(D, I, E, top, shared, n, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    names = ("gate", "up", "down")
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        hidden_size=D, expert_size=I, experts=E, top=top, prefix="f.", activation="silu_gated", scores="sigmoid", correction=False, weight_input=True,
        shared_gate="shared.sg", shared=dict(intermediate_size=shared, prefix="f.shared.", names=names) if shared else None)), dtype=dt, device=DEV)
    w = draw(part, 71)
    for k in w:
        if k.endswith(("gate", "up")):
            w[k] = 2.0 * w[k]
    w["f.router"] = 3.0 * D ** -0.5 * w["f.router"]           # scores that differ and stay away from one
    load(part, w, dt)
    wh = hold(part, w, dt)
    x = held(rand((n, D), 77), dt)
    mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
    margins = []
    want = P.moe_ff(x, wh, "f.", mlp, torch.float64, margins)
    idx, weights, _ = P.route(x, wh, "f.", top, torch.float64)
    outside = torch.zeros_like(want)                     # the weights at the outputs instead: another function
    for j in range(top):
        outside += torch.stack([weights[t, j] * P.gated_ff(x[t:t + 1], wh, f"f.e{int(idx[t, j])}.", torch.float64)[0] for t in range(n)])
    plain = P.moe_ff(x, wh, "f.", dict(mlp, shared=None), torch.float64)
    assert (outside - plain).abs().max() > 0.05 * plain.abs().max()
    sure = margins[0] > 1e-3
    assert sure.sum() >= n // 2
    got = run_ff(part, x, dt)
    assert_close(got[sure.to(DEV)], want[sure], dt, "experts", 2e-5 if dt == torch.float32 else 0.04)


def test_scores_that_round_to_one_are_told_apart():
    """Logits of 20 to 27: their sigmoids are one number in 32 bits, the choice is still by the largest."""
    from vllm_oxide_b200 import kernels
    E, W, n = 8, 32, 5
    x = torch.zeros((n, W), device=DEV)
    x[:, 0] = 1.0
    r = torch.zeros((E, W), device=DEV)
    r[:, 0] = 20.0 + torch.tensor([3.0, 1.0, 7.0, 2.0, 6.0, 0.0, 5.0, 4.0], device=DEV)
    ids, weights = torch.empty((n, 3), dtype=torch.int32, device=DEV), torch.empty((n, 3), device=DEV)
    kernels.moe_route(x, r, None, ids, weights, n, 3, 1, 1, sigmoid_scores=True)
    assert ids[0].tolist() == [2, 4, 6] and bool((weights == 1.0).all())


# ---------------------------------------------------------------- sublayers that end in the stream
@pytest.mark.parametrize("M", [1, 5, 8, 9, 16])
@pytest.mark.parametrize("N, K", [(64, 128), (100, 320), (4800, 64), (33, 256)])
def test_a_product_that_ends_in_the_stream(M, N, K):
    """The weight-streaming product added into a float stream, unrounded, with the norm that follows beside it, or without."""
    from vllm_oxide_b200 import kernels
    bf, f32 = torch.bfloat16, torch.float32
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    x, w = rand((M, K), 1).to(bf).to(DEV), rand((N, K), 2, K ** -0.5).to(bf).to(DEV)
    s0, g, b = rand((M, N), 3, 2.0).float(), (1.0 + 0.3 * rand((N,), 4)).float(), rand((N,), 5, 0.3).float()
    alpha = torch.tensor([0.6])
    want = s0.double() + x.double().cpu() @ w.double().cpu().T
    for bias in (b, None):
        stream, normed = s0.to(DEV), torch.empty((M, N), dtype=bf, device=DEV)
        kernels.gemm_skinny(x, w, stream, kernels.EPI_STREAM, err, emit_tanh=(alpha.to(DEV), g.to(DEV), None if bias is None else b.to(DEV), normed))
        assert_close(stream, want, f32, "stream", 1e-5)
        assert_close(normed, P.tanh_norm(want, alpha.double(), g.double(), b.double() if bias is not None else 0.0), bf, "normed", 0.005)
    stream = s0.to(DEV)
    kernels.gemm_skinny(x, w, stream, kernels.EPI_STREAM, err)
    assert_close(stream, want, f32, "stream, no norm", 1e-5)
    assert int(err.item()) == 0


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T, D, top", [(3, 64, 4), (7, 30, 2), (5, 1028, 1), (2, 4100, 9), (300, 128, 3)])
def test_a_sum_of_experts_that_ends_in_the_stream(T, D, top, dt):
    from vllm_oxide_b200 import kernels
    f32 = torch.float32
    dev = lambda t, d=f32: t.to(d).to(DEV).contiguous()
    y, wt, add, ag = rand((T * top + 3, D), 1), rand((T, top), 2), held(rand((T, D), 3), dt), rand((T,), 4)
    y, wt, ag = y.float().double(), wt.float().double(), ag.float().double()
    slot = torch.randperm(T * top + 3, generator=torch.Generator().manual_seed(5))[:T * top].int()
    slot[1] = -1                                                              # a pair that has no row
    s0, g, b, alpha = rand((T, D), 6).float(), (1.0 + 0.3 * rand((D,), 7)).float(), rand((D,), 8, 0.3).float(), torch.tensor([0.8])
    rows = torch.where((slot >= 0)[:, None], y[slot.long().clamp(min=0)], torch.zeros(1, dtype=torch.float64)).reshape(T, top, D)
    for weights, gate in ((wt, ag), (None, ag), (wt, None)):
        total = ((rows * weights[..., None]) if weights is not None else rows).sum(1) + add * (gate[:, None] if gate is not None else 1.0)
        args = (dev(y), slot.to(DEV), None if weights is None else dev(weights))
        more = dict(add=dev(add, dt), add_gate=None if gate is None else dev(gate))
        out = torch.empty((T, D), dtype=dt, device=DEV)
        kernels.moe_combine(*args, out, T, top, **more)
        assert_close(out, total, dt, "a row of its own", 3e-6 if dt == f32 else 0.01)
        stream = dev(s0)
        kernels.moe_combine(*args, out, T, top, stream=stream, norm=(dev(alpha), dev(g), dev(b)), **more)
        assert_close(stream, s0.double() + total, f32, "stream", 3e-6)
        assert_close(out, P.tanh_norm(s0.double() + total, alpha.double(), g.double(), b.double()), dt, "normed", 3e-6 if dt == f32 else 0.005)
        stream = dev(s0)
        kernels.moe_combine(*args, None, T, top, stream=stream, **more)
        assert_close(stream, s0.double() + total, f32, "stream, no norm", 3e-6)
