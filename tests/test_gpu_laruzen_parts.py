"""Every mechanism of Laruzen alone, as a part with pages and state slots of its own, against its plain function
(tests/plain/laruzen_plain.py): the pair embedding, the stream's step with its norms and the token shift, both linear
attentions at every width of their scan (whole, in portions, cut along the tokens), attention with normed heads and values and
a learned sink on the plain and on the tensor-core kernels, the recurrent block, the gelu-gated feed-forward, experts beside a
shared one, the pair of mixers."""
import pytest
import torch

from helpers import DEV, Alone, assert_close, held, make_context, rand
from plain import laruzen_plain as P

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5


def load(part, w, dt):
    """Gives a part the tensors it lists, each in the type the engine keeps it in."""
    from vllm_oxide_b200.weights.loader import kept_dtype
    part.load({s.name: w[s.name].to(kept_dtype(s.role, dt)).to(DEV).contiguous() for s in part.tensor_specs()})


def draw(part, seed, rank=None):
    """Random tensors for everything the part lists (float64): matrices by their fan-in, gains near one, the rest small.  `rank`:
    what a size that is read from the tensors is here."""
    w = {}
    for i, s in enumerate(part.tensor_specs()):
        shape = tuple(rank if n < 0 else n for n in s.shape)
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


# ---------------------------------------------------------------- what opens the stream
@pytest.mark.parametrize("dt", DTYPES)
def test_pair_embedding_over_requests_and_slots_used_again(dt):
    from vllm_oxide_b200.cache.paged_cache import PagedCache
    from vllm_oxide_b200.parts import PartSpec, build_part
    V, D, buckets, mp, mc = 50, 44, 23, 1000003, 77
    part = build_part("embedding", PartSpec("pair_embedding", dict(vocab_size=V, size=D, table_name="e", pair_name="p", buckets=buckets,
                                                                   mul_prev=mp, mul_cur=mc)), dtype=dt, device=DEV)
    w = {"e": rand((V, D), 1), "p": rand((buckets + 1, D), 2)}
    load(part, w, dt)
    W = {"embed": held(w["e"], dt), "bigram": held(w["p"], dt)}
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    cache = PagedCache([None], [part.state_spec()], dt, DEV, 16, 40, 2)
    toks = {r: torch.randint(0, V, (n,), generator=torch.Generator().manual_seed(r)).tolist() for r, n in ((1, 40), (2, 9), (3, 17), (4, 1))}
    want = {r: P.embedded(cfg, W, t, torch.float64) for r, t in toks.items()}
    at = {r: 0 for r in toks}
    # portions of one request beside single tokens of another; requests 3 and 4 find the slots of 1 and 2
    for portions in [[(1, 7)], [(1, 1), (2, 3)], [(2, 1), (1, 2)], [(1, 30), (2, 5)], [(3, 1), (4, 1)], [(3, 16)]]:
        for r, _ in portions:
            if at[r] == 0:
                assert cache.manager.add_request(r)
            cache.manager.ensure(r, at[r], 40)
        ctx = make_context(cache.manager, [(r, at[r], toks[r][at[r]:at[r] + n], []) for r, n in portions], dt)
        cache.zero_states([int(s) for s, f in zip(ctx.host_view("state_slots"), ctx.host_view("state_fresh")) if f])
        hidden, stream = part.open(ctx, cache.states[0])
        assert hidden is None and stream.dtype == torch.float32 and int(ctx.err.item()) == 0
        k = 0
        for r, n in portions:
            # two 16-bit numbers' sum, unrounded
            assert torch.allclose(stream[k:k + n].double().cpu(), want[r][at[r]:at[r] + n], rtol=1e-6, atol=1e-6), (r, at[r])
            k += n
            at[r] += n
            if at[r] == len(toks[r]):
                cache.manager.free_request(r)


# ---------------------------------------------------------------- the stream's step with norms and shift
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D", [8, 30, 64, 516, 1040, 2052, 4100, 8196])
def test_norms_around_the_stream(D, dt):
    """residual_norm_step at every width of its kernels: rows in registers, and in shared memory where the width does not allow."""
    from vllm_oxide_b200 import kernels
    n = 5
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = lambda t, d=dt: t.to(d).to(DEV).contiguous()
    x, y, inj = rand((n, D), 1).float().double(), held(rand((n, D), 2, 3.0), dt), rand((n, D), 6).float().double()
    wp, wq = ((1.0 + 0.3 * rand((D,), s)).float().double() for s in (3, 4))
    stream, out = dev(x, torch.float32), torch.empty((n, D), dtype=dt, device=DEV)
    keep = torch.empty((n, D), dtype=torch.float32, device=DEV)
    kernels.residual_norm_step(stream, EPS, err, y=dev(y), w_post=dev(wp, torch.float32), inject=dev(inj, torch.float32), keep=keep,
                               w_pre=dev(wq, torch.float32), out=out)
    want = x + P.rms(y, EPS) * wp + inj
    assert_close(stream, want, torch.float32, "stream", 1e-6)
    assert torch.equal(keep, stream)
    assert_close(out, P.rms(want, EPS) * wq, dt, "normed")
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
    some, before = torch.empty((3, D), dtype=dt, device=DEV), stream.clone()
    kernels.residual_norm_step(stream, EPS, err, y=dev(y), w_post=dev(wp, torch.float32), w_pre=dev(wq, torch.float32), out=some, rows=rows, n_out=3)
    assert torch.equal(stream, before) and int(err.item()) == 0
    assert_close(some, (P.rms(want + P.rms(y, EPS) * wp, EPS) * wq)[[4, 0, 4]], dt, "chosen rows")
    kernels.residual_norm_step(stream, EPS, err, y=dev(y), init=True)
    assert_close(stream, y, torch.float32, "a stream that begins", 1e-6)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D, lengths", [(8, (9, 1, 4)), (30, (3, 5)), (64, (1, 1, 1)), (516, (40, 2, 1, 7)), (1040, (6, 1)), (2052, (5, 1, 3)),
                                        (4100, (3, 4)), (8196, (2, 1, 3)), (72, (1500, 1, 7, 2000)), (42, (1300, 1, 1400))])
def test_norms_and_token_shift(D, lengths, dt):
    """Two steps of portions: the h before a portion's first token comes from the slot, the last is left there; long portions are
    walked by several blocks, each of which makes the h before its first token again."""
    from vllm_oxide_b200 import kernels
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = lambda t, d=dt: t.to(d).to(DEV).contiguous()
    f32 = torch.float32
    n, B = sum(lengths), len(lengths)
    wp, wq = ((1.0 + 0.3 * rand((D,), s)).float().double() for s in (3, 4))
    shift = torch.sigmoid(rand((D,), 5)).float().double()
    state = torch.full((B + 1, D + 3), 55.0, dtype=f32, device=DEV)      # rows wider than the part, a slot nobody uses
    slots = list(range(B, 0, -1))
    cu = torch.tensor([0] + list(torch.tensor(lengths).cumsum(0)), dtype=torch.int32, device=DEV)
    req = torch.tensor(sum(([b] * m for b, m in enumerate(lengths)), []) + [-1, -1], dtype=torch.int32, device=DEV)    # two padding rows
    slot_t = torch.tensor(slots, dtype=torch.int32, device=DEV)
    last = torch.zeros((B, D), dtype=torch.float64)
    state[1:, :D] = 0.0
    for step in range(2):
        x, y = rand((n + 2, D), 10 + step).float().double(), held(rand((n + 2, D), 20 + step, 2.0), dt)
        stream, new = dev(x, f32), torch.full((n + 2, D), 9.0, dtype=f32, device=DEV)
        out = torch.empty((n + 2, D), dtype=dt, device=DEV)
        has_y = step == 0 or D != 64
        kernels.residual_norm_shift_step(stream, new, EPS, err, dev(y) if has_y else None, dev(wp, f32) if has_y else None, dev(wq, f32),
                                         dev(shift, f32), state[:, :], req, cu, slot_t, out)
        xs = x + P.rms(y, EPS) * wp if has_y else x
        assert torch.equal(stream, dev(x, f32)) and int(err.item()) == 0
        if has_y:
            assert_close(new, xs, f32, "the new stream", 1e-6)
        h = P.rms(xs, EPS) * wq
        want, at = h.clone(), 0
        for b, m in enumerate(lengths):
            prev = torch.cat([last[b:b + 1], h[at:at + m - 1]])
            want[at:at + m] = h[at:at + m] + (prev - h[at:at + m]) * shift
            last[b] = h[at + m - 1]
            at += m
        assert_close(out, want, dt, f"step {step}", 3e-6 if dt == f32 else None)
        assert_close(state[slot_t.long(), :D], last, f32, f"the last rows after step {step}", 3e-6)
    assert bool((state[0] == 55.0).all()) and bool((state[:, D:] == 55.0).all())


# ---------------------------------------------------------------- linear attention
SCANS = [(3, 16, 8), (2, 24, 20), (1, 32, 32), (5, 12, 40), (2, 64, 48), (3, 128, 12), (1, 200, 36), (2, 8, 1), (1, 1, 16), (2, 128, 128)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", SCANS)
def test_gated_linear_attention(heads, dim, vdim, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, tau, rank = (64, 7.0, 70) if dim == 64 else (40, 16.0, 5)
    part = build_part("mixer", PartSpec("gated_linear_attention", dict(hidden_size=D, num_heads=heads, dim=dim, vdim=vdim, tau=tau, eps=EPS,
                                                                       prefix="m.")), dtype=dt, device=DEV)
    w = draw(part, 11, rank)
    w["m.a2"] = 2.0 * w["m.a2"]
    w["m.a2.b"] = 3.0 * w["m.a2.b"] + 1.0       # channels that forget at rates of their own, some all but never, some at once
    load(part, w, dt)
    assert part.rank == rank
    x = held(rand((330, D), 5), dt)
    want = P.gla(x, hold(part, w, dt), "m.", dict(heads=heads, dim=dim, vdim=vdim, tau=tau), EPS, torch.float64)
    run_cuts(part, x, [[330], [290] + [1] * 40, [7, 2, 33, 90], [2]], want, dt, f"gla {heads} x {dim} x {vdim}", 5e-5 if dt == torch.float32 else 0.04)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", [s for s in SCANS if s[2] > 1] + [(5, 8, 1), (6, 24, 100)])
def test_lightning_attention(heads, dim, vdim, dt):
    """(The last: a row of all heads that the wide norm kernel takes.)"""
    from vllm_oxide_b200.parts import PartSpec, build_part
    D = 40
    decay = [0.999 - 0.3 * h for h in range(min(heads, 3))] + [0.0, 1.0, 0.5][:max(0, heads - 3)]
    part = build_part("mixer", PartSpec("lightning_attention", dict(hidden_size=D, num_heads=heads, dim=dim, vdim=vdim, decay=decay, eps=EPS,
                                                                    prefix="m.")), dtype=dt, device=DEV)
    w = draw(part, 31)
    load(part, w, dt)
    x = held(rand((330, D), 6), dt)
    want = P.lightning(x, hold(part, w, dt), "m.", dict(heads=heads, dim=dim, vdim=vdim, decay=decay), EPS, torch.float64)
    run_cuts(part, x, [[330], [290] + [1] * 40, [7, 2, 33, 90], [2]], want, dt, f"lightning {heads} x {dim} x {vdim}",
             5e-5 if dt == torch.float32 else 0.04)


@pytest.mark.parametrize("kind", ["gated_linear_attention", "lightning_attention"])
def test_a_state_that_never_forgets(kind):
    """With decays of all but one, the last rows hang on what the first tokens wrote, in every cut."""
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, m = 32, dict(heads=2, dim=48, vdim=24)
    more = dict(tau=64.0) if kind.startswith("gated") else dict(decay=[1.0, 0.9999])
    part = build_part("mixer", PartSpec(kind, dict(hidden_size=D, num_heads=2, dim=48, vdim=24, eps=EPS, prefix="m.", **more)), dtype=torch.float32,
                      device=DEV)
    w = draw(part, 3, 4)
    if kind.startswith("gated"):
        w["m.a2.b"] = w["m.a2.b"] + 9.0
    load(part, w, torch.float32)
    plain = P.gla if kind.startswith("gated") else P.lightning
    x = held(rand((700, D), 7), torch.float32)
    want = plain(x, hold(part, w, torch.float32), "m.", dict(m, **more), EPS, torch.float64)
    other = x.clone()
    other[:10] = rand((10, D), 8, 3.0)
    gap = (plain(other, hold(part, w, torch.float32), "m.", dict(m, **more), EPS, torch.float64) - want)[-1].abs().max()
    assert gap > 0.02 * want[-1].abs().max()
    run_cuts(part, x, [[700], [400] + [3] * 100, [650] + [1] * 50], want, torch.float32, kind, 1e-4, pages=60)


# ---------------------------------------------------------------- attention
YARN = {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 2.0}
ATTENTION = {
    # (D, sizes, fast in 16 bits): padded to 48, 64 and 128 (TMA, tcgen05), 32 (cp.async); more query heads than those kernels take
    "values wider than keys": (40, dict(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.3, mask={"size": 19}, rot={"dims": 16, "base": 100.0, "scaling": YARN}), True),
    "64 wide, the whole head turns": (64, dict(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.15, mask={"size": 44}, rot={"dims": 64, "base": 1e4, "scaling": YARN}), True),
    "128 wide, a window of one tile": (48, dict(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.1, mask={"size": 64}, rot={"dims": 32, "base": 1e4}), True),
    "keys wider than values": (32, dict(heads=3, kv_heads=3, dim=40, vdim=16, scale=0.25, mask={"size": 23}, rot={"dims": 10, "base": 777.0, "scaling": YARN}), True),
    "a window of one, one head": (32, dict(heads=1, kv_heads=1, dim=16, vdim=32, scale=0.3, mask={"size": 1}, rot={"dims": 16, "base": 50.0}), True),
    "no window, no rotation": (32, dict(heads=6, kv_heads=2, dim=16, vdim=16, scale=0.3, mask=None, rot=None), True),
    "odd sizes": (32, dict(heads=2, kv_heads=1, dim=9, vdim=7, scale=0.5, mask={"size": 33}, rot={"dims": 6, "base": 60.0}), True),
    "twenty heads on one": (32, dict(heads=20, kv_heads=1, dim=16, vdim=16, scale=0.3, mask={"size": 50}, rot={"dims": 8, "base": 1e4}), False),
}


def attention_part(dt, D, m, **options):
    from vllm_oxide_b200.parts import PartSpec, build_part
    rot, positions, position = m.get("rot"), {}, None
    if rot:
        position = "r"
        positions["r"] = build_part("position", PartSpec("rope", dict(head_dim=m["dim"], rotary_dim=rot["dims"], max_position=1 << 30,
                                                                      theta=rot["base"], interleaved=False, table=False, precise=True,
                                                                      scaling=rot.get("scaling"))), device=DEV)
    return build_part("mixer", PartSpec("attention_normed", dict(
        hidden_size=D, num_heads=m["heads"], num_kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], eps=EPS, prefix="m.",
        window=(m.get("mask") or {}).get("size"), position=position, **options)), positions=positions, dtype=dt, device=DEV)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", sorted(ATTENTION))
def test_attention_with_normed_heads_and_a_learned_sink(case, dt):
    D, m, fast = ATTENTION[case]
    part = attention_part(dt, D, m)
    w = draw(part, 21)
    w["m.sink"] = 2.0 * rand((m["heads"],), 99) + torch.arange(m["heads"], dtype=torch.float64) % 3     # sinks that count, each its own
    load(part, w, dt)
    x = held(rand((200, D), 6), dt)
    wh = hold(part, w, dt)
    want = P.window_attention(x, wh, "m.", m, EPS, torch.float64)
    without = P.window_attention(x, dict(wh, **{"m.sink": wh["m.sink"] - 50.0}), "m.", m, EPS, torch.float64)
    assert (without - want).abs().max() > 0.1 * want.abs().max(), "the sinks count"
    ran = {}
    run_cuts(part, x, [[200], [150] + [1] * 50, [7, 2, 33, 64], [2]], want, dt, case, kernels_ran=ran)
    if dt == torch.bfloat16 and fast:
        assert "paged_attention_generic" not in ran and any(k.startswith("attention_prefill") for k in ran) and \
            any(k.startswith("attention_decode") for k in ran), ran
    else:
        assert "paged_attention_generic" in ran


@pytest.mark.parametrize("dt", DTYPES)
def test_attention_options_left_out(dt):
    """Without biases, head norms, value norm, sink and gate it is the plain windowed attention."""
    D, m = 48, dict(heads=4, kv_heads=2, dim=32, vdim=32, scale=0.2, mask={"size": 30}, rot=None)
    part = attention_part(dt, D, m, bias=False, qk_norm=False, value_norm=False, sink=False, gate=False)
    assert {s.name for s in part.tensor_specs()} == {"m.q", "m.k", "m.v", "m.o"}
    w = draw(part, 5)
    load(part, w, dt)
    wh = hold(part, w, dt)
    x = held(rand((90, D), 6), dt)
    q, k, v = (x @ wh["m." + n].T for n in "qkv")
    s = torch.einsum("ihd,jhd->hij", q.reshape(90, 4, 32), k.reshape(90, 2, 32).repeat_interleave(2, 1)) * 0.2
    i, j = torch.arange(90)[:, None], torch.arange(90)[None, :]
    a = torch.softmax(s.masked_fill(~((j <= i) & (i - j < 30)), float("-inf")), -1)
    want = torch.einsum("hij,jhd->ihd", a, v.reshape(90, 2, 32).repeat_interleave(2, 1)).reshape(90, 128) @ wh["m.o"].T
    run_cuts(part, x, [[90], [60] + [1] * 30, [2, 17]], want, dt, "plain options")


@pytest.mark.parametrize("sink", [-60.0, -8.0, 0.0, 9.0, 60.0])
def test_sinks_far_below_and_above_the_scores(sink):
    """A sink that towers over the scores leaves nothing of a head, one far below them changes nothing; no number overflows."""
    D, m = 32, dict(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.3, mask={"size": 40}, rot=None)
    for dt in DTYPES:
        part = attention_part(dt, D, m)
        w = draw(part, 8)
        w["m.sink"] = torch.tensor([sink, sink + 1.0, sink, 0.5], dtype=torch.float64)
        load(part, w, dt)
        x = held(rand((100, D), 9), dt)
        want = P.window_attention(x, hold(part, w, dt), "m.", m, EPS, torch.float64)
        run_cuts(part, x, [[100], [80] + [1] * 20], want, dt, f"sink {sink}")


# ---------------------------------------------------------------- the recurrent block
RECURRENT = [(40, 36, 3, 5), (48, 64, 1, 4), (32, 33, 11, 2), (64, 128, 2, 4), (40, 20, 20, 1), (24, 7, 1, 9), (64, 512, 2, 3)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D, width, blocks, taps", RECURRENT)
def test_recurrent_block(D, width, blocks, taps, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    part = build_part("mixer", PartSpec("recurrent_block", dict(hidden_size=D, width=width, blocks=blocks, taps=taps, prefix="m.")), dtype=dt,
                      device=DEV)
    w = draw(part, 41)
    w["m.lam"] = 2.0 * w["m.lam"] - 4.0          # channels that forget slowly, each at a rate of its own
    w["m.x.b"] = 3.0 * w["m.x.b"]                 # a bias in front of the filter shows in the first tokens, whose window holds zeros
    load(part, w, dt)
    x = held(rand((330, D), 8), dt)
    want = P.recurrent_block(x, hold(part, w, dt), "m.", dict(width=width, blocks=blocks), EPS, torch.float64)
    run_cuts(part, x, [[330], [290] + [1] * 40, [3, 1, 17, 2, 90], [2], [8, 9]], want, dt, f"{width} channels in {blocks} parts, {taps} taps",
             5e-5 if dt == torch.float32 else 0.04)


@pytest.mark.parametrize("n", [600, 1500])
def test_slow_channels_write_what_they_should(n):
    """A decay of one minus 1e-6: 1 - a^2 as a difference of floats would be off by percents.  (1,500 tokens: the most ranges.)"""
    from vllm_oxide_b200.parts import PartSpec, build_part
    D, W = 24, 32
    part = build_part("mixer", PartSpec("recurrent_block", dict(hidden_size=D, width=W, blocks=2, taps=3, prefix="m.")), dtype=torch.float32,
                      device=DEV)
    w = draw(part, 51)
    w["m.lam"] = torch.linspace(-16.0, 4.0, W, dtype=torch.float64)
    load(part, w, torch.float32)
    x = held(rand((n, D), 9), torch.float32)
    want = P.recurrent_block(x, hold(part, w, torch.float32), "m.", dict(width=W, blocks=2), EPS, torch.float64)
    run_cuts(part, x, [[n], [100, 1, 7]], want, torch.float32, "slow channels", 5e-5, pages=100)


# ---------------------------------------------------------------- two mixers side by side, pages and slots used again
@pytest.mark.parametrize("dt", DTYPES)
def test_pages_and_slots_used_again_by_the_pair(dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    D = 48
    left = PartSpec("attention_normed", dict(hidden_size=D, num_heads=2, num_kv_heads=1, dim=16, vdim=24, scale=0.3, eps=EPS, prefix="m.left.",
                                             window=20, position=None))
    right = PartSpec("recurrent_block", dict(hidden_size=D, width=40, blocks=2, taps=4, prefix="m.right."))
    part = build_part("mixer", PartSpec("side_by_side", dict(left=left, right=right, hidden_size=D, eps=EPS, left_norm="m.left.out",
                                                             right_norm="m.right.out")), positions={}, dtype=dt, device=DEV)
    w = draw(part, 31)
    w["m.left.o.b"] = 2.0 * w["m.left.o.b"]       # enters in front of the left side's norm
    w["m.right.lam"] = w["m.right.lam"] - 4.0
    load(part, w, dt)
    wh = hold(part, w, dt)
    m = {"left": dict(heads=2, kv_heads=1, dim=16, vdim=24, scale=0.3, mask=dict(size=20)), "right": dict(width=40, blocks=2)}
    alone = Alone([part], dt, block_size=16, pages=9, slots=2)
    xs = {rid: held(rand((n, D), 40 + rid), dt) for rid, n in ((1, 100), (2, 37), (3, 64), (4, 5), (5, 90))}
    got, at = {rid: [] for rid in xs}, {rid: 0 for rid in xs}
    for portions in [[(1, 50)], [(1, 1), (2, 30)], [(1, 49), (2, 7)], [(3, 64)], [(4, 5), (5, 2)], [(5, 88)]]:
        batch = [(rid, xs[rid][at[rid]:at[rid] + n]) for rid, n in portions]
        out = alone.step(batch, end=[rid for rid, n in portions if at[rid] + n == xs[rid].shape[0]])[0]
        k = 0
        for rid, rows in batch:
            got[rid].append(out[k:k + rows.shape[0]])
            at[rid] += rows.shape[0]
            k += rows.shape[0]
    assert alone.m.num_free_blocks(0) == 9 and alone.m.num_free_state_slots == 2
    for rid, x in xs.items():
        assert_close(torch.cat(got[rid]), P.side_by_side(x, wh, "m.", m, EPS, torch.float64), dt, f"request {rid}",
                     3e-5 if dt == torch.float32 else 0.04)


# ---------------------------------------------------------------- feed-forwards
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
@pytest.mark.parametrize("D, I, n", [(64, 96, 5), (128, 192, 40), (48, 37, 9), (40, 24, 3), (64, 8, 16)])
def test_gelu_gated_feed_forward(D, I, n, dt):
    """As the epilogue of the weight-streaming product (few tokens, a width that is a multiple of 64) and as a kernel of its own."""
    from vllm_oxide_b200.parts import PartSpec, build_part
    part = build_part("feed_forward", PartSpec("swiglu", dict(hidden_size=D, intermediate_size=I, prefix="f.", names=("gate", "up", "down"),
                                                              activation="gelu_tanh")), dtype=dt, device=DEV)
    w = draw(part, 61)
    load(part, w, dt)
    x = held(rand((n, D), 7, 2.0), dt)
    wh = hold(part, w, dt)
    want = P.gated_ff(x, wh, "f.", P.gelu_tanh, torch.float64)
    assert (P.gated_ff(x, wh, "f.", P.silu, torch.float64) - want).abs().max() > 0.03 * want.abs().max()
    assert_close(run_ff(part, x, dt), want, dt, "gelu gate")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D, I, E, top, shared, n", [
    (64, 24, 12, 2, 40, 40),         # few pairs: the experts' rows are streamed pair by pair in bfloat16
    (48, 16, 6, 6, 8, 9),            # every expert chosen
    (40, 8, 5, 1, 24, 5),            # one expert: its weight is one
    (128, 64, 8, 4, 64, 300),        # enough pairs for the tcgen05 products in bfloat16
    (72, 33, 4, 2, 17, 3),           # odd widths: the float-accumulating tile kernel
    (64, 24, 1, 1, 40, 7),           # a single expert
    (64, 24, 7, 3, 0, 20),           # no shared expert
])
def test_experts_beside_a_shared_one(D, I, E, top, shared, n, dt):
    from vllm_oxide_b200.parts import PartSpec, build_part
    names = ("gate", "up", "down")
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        hidden_size=D, expert_size=I, experts=E, top=top, prefix="f.", activation="silu_gated", scores="softmax", correction=False,
        normalise=True, shared=dict(intermediate_size=shared, prefix="f.shared.", names=names) if shared else None)), dtype=dt, device=DEV)
    w = draw(part, 71)
    w["f.router"] = 2.0 * w["f.router"]
    load(part, w, dt)
    wh = hold(part, w, dt)
    x = held(rand((n, D), 77), dt)
    mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
    margins = []
    want = P.moe_ff(x, wh, "f.", mlp, torch.float64, margins)
    sure = margins[0] > 1e-3
    assert sure.sum() >= n // 2
    got = run_ff(part, x, dt)
    assert_close(got[sure.to(DEV)], want[sure], dt, "experts", 2e-5 if dt == torch.float32 else 0.04)
