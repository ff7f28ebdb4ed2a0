"""Plain, slow Laruzen forward pass: whole sequences, no cache, one function per mechanism.

The oracle for the engine's Laruzen model.  It shares no code with the package: it reads a model folder with its own
few lines (or takes a dict of tensors), works on one whole sequence at a time and keeps nothing between calls.  Every
function works in the dtype `dt` it is given (float64 for an oracle); nothing is rounded below `dt`.

Notation: n tokens, D the model width.  N(x) = x / rms(x) * (1 + w).  A layer is

    h = N1(x);  h_t <- h_t + (h_{t-1} - h_t) * shift;   x += N1b(mixer(h));   x += N2b(ff(N2(x)))

with h_{-1} = 0.  x starts as a token's embedding plus the embedding of the pair (token before, token), hashed into
buckets.  The mixer is `gla` (a matrix state per head with a decay per key channel), `lightning` (a matrix state per head
with one fixed decay) or `parallel` (windowed attention with normed, partly rotated heads, normed values, a learned sink
and an output gate, beside a gated linear recurrence behind a short convolution; each side normed, half their sum).
The feed-forward is a gated layer (tanh-form gelu), or a mixture of gated SiLU experts beside a shared one.
"""
import json
import math
import struct

import torch

_ST = {"F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16, "F64": torch.float64,
       "I32": torch.int32, "I64": torch.int64}


def read_folder(path):
    with open(f"{path}/config.json") as f:
        cfg = json.load(f)
    with open(f"{path}/model.safetensors", "rb") as f:
        blob = f.read()
    (n,) = struct.unpack("<Q", blob[:8])
    head = json.loads(blob[8:8 + n])
    out = {}
    for name, meta in head.items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        t = torch.frombuffer(bytearray(blob[8 + n + a:8 + n + b]), dtype=_ST[meta["dtype"]])
        out[name] = t.reshape(meta["shape"]).clone()
    return cfg, out


# ---------------------------------------------------------------- small functions
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(x):
    return torch.where(x > 30.0, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


# ---------------------------------------------------------------- embedding
def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """The row of the pair table every token reads; the first token of a sequence reads the extra row `buckets`."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows


def embedded(cfg, W, tokens, dt):
    x = W["embed"].to(dt)[torch.as_tensor(list(tokens), dtype=torch.long)]
    b = cfg["embedding"].get("bigram") if cfg.get("embedding") else None
    if b:
        rows = bigram_rows(list(tokens), int(b["mul_prev"]), int(b["mul_cur"]), int(b["buckets"]))
        x = x + W["bigram"].to(dt)[torch.as_tensor(rows, dtype=torch.long)]
    return x


def token_shift(h, w):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    return h + (before - h) * w


# ---------------------------------------------------------------- matrix-state recurrences
def matrix_recurrence(q, k, v, decay):
    """q, k [n, H, dk], v [n, H, dv], decay [n, H, dk] (rows of the state): o [n, H, dv]."""
    n, H, dk = q.shape
    S = q.new_zeros((H, dk, v.shape[2]))
    out = q.new_zeros((n, H, v.shape[2]))
    for t in range(n):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def gla(h, W, p, m, eps, dt):
    n = h.shape[0]
    H, dk, dv, tau = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"])
    g = lambda name: W[p + name].to(dt)
    q = (h @ g("q").T).reshape(n, H, dk) * dk ** -0.5
    k = (h @ g("k").T).reshape(n, H, dk)
    v = (h @ g("v").T).reshape(n, H, dv)
    z = (h @ g("a1").T) @ g("a2").T + g("a2.b")
    alpha = sigmoid(z) ** (1.0 / tau)
    o = matrix_recurrence(q, k, v, alpha.reshape(n, H, dk))
    o = (rms(o, eps) * g("norm")).reshape(n, H * dv)
    return (o * silu(h @ g("g").T)) @ g("o").T


def lightning(h, W, p, m, eps, dt):
    n = h.shape[0]
    H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda name: W[p + name].to(dt)
    q = silu(h @ g("q").T).reshape(n, H, dk)
    k = silu(h @ g("k").T).reshape(n, H, dk)
    v = silu(h @ g("v").T).reshape(n, H, dv)
    decay = torch.tensor([float(d) for d in m["decay"]], dtype=dt)[None, :, None].expand(n, H, dk)
    o = matrix_recurrence(q, k, v, decay).reshape(n, H * dv)
    o = rms(o, eps) * g("norm")
    return (o * sigmoid(h @ g("g").T)) @ g("o").T


# ---------------------------------------------------------------- the left side: attention
def stretched_frequencies(dims, base, scaling, dt=torch.float64):
    """f_i of pair i (i < dims / 2) and the amplitude of cos and sin."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=dt)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    where = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(where(float(scaling["fast"]))), 0)
    hi = min(math.ceil(where(float(scaling["slow"]))), dims - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(half)], dtype=dt)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_front_halves(x, rot, dt):
    """x [n, heads, dim]: among the first rot.dims elements, i turns with i + dims/2; the rest stays."""
    dims = int(rot["dims"]) if rot else 0
    if dims == 0:
        return x
    freq, amp = stretched_frequencies(dims, float(rot["base"]), rot.get("scaling"), dt)
    half = dims // 2
    ang = torch.arange(x.shape[0], dtype=dt)[:, None] * freq[None, :]
    c, s = (torch.cos(ang) * amp)[:, None, :], (torch.sin(ang) * amp)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def window_attention(h, W, p, m, eps, dt):
    n = h.shape[0]
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda name: W[p + name].to(dt)
    q = (h @ g("q").T + g("q.b")).reshape(n, H, dk)
    k = (h @ g("k").T + g("k.b")).reshape(n, G, dk)
    v = (h @ g("v").T + g("v.b")).reshape(n, G, dv)
    q = rotate_front_halves(rms(q, eps) * g("q.norm"), m.get("rot"), dt)
    k = rotate_front_halves(rms(k, eps) * g("k.norm"), m.get("rot"), dt)
    v = rms(v, eps)
    kh = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, kh]) * float(m["scale"])
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    size = int((m.get("mask") or {}).get("size") or 0)
    see = (j <= i) & (i - j < size) if size else (j <= i)
    s = s.masked_fill(~see, float("-inf"))
    sink = g("sink")[:, None, None].expand(H, n, 1)
    a = torch.softmax(torch.cat([s, sink], dim=-1), dim=-1)[..., :-1]
    o = torch.einsum("hij,jhd->ihd", a, v[:, kh]).reshape(n, H * dv)
    o = o * sigmoid(h @ g("g").T)
    return o @ g("o").T + g("o.b")


# ---------------------------------------------------------------- the right side: gated linear recurrence
def causal_conv(u, w, b):
    """y[t] = b + sum_j w[:, j] u[t - taps + 1 + j], zeros before the start.  u [n, C], w [C, taps]."""
    n, taps = u.shape[0], w.shape[1]
    pad = torch.cat([u.new_zeros((taps - 1, u.shape[1])), u], dim=0)
    y = torch.zeros_like(u) + b
    for j in range(taps):
        y = y + pad[j:j + n] * w[:, j]
    return y


def linear_recurrence(u, W, p, m, dt):
    """S [n, width] of the recurrence over u [n, width]."""
    n, width = u.shape
    blocks = int(m["blocks"])
    g = lambda name: W[p + name].to(dt)
    ub = u.reshape(n, blocks, width // blocks)
    r = sigmoid(torch.einsum("nbi,boi->nbo", ub, g("ra")) + g("ra.b")).reshape(n, width)
    i = sigmoid(torch.einsum("nbi,boi->nbo", ub, g("ri")) + g("ri.b")).reshape(n, width)
    log_a = -8.0 * r * softplus(g("lam"))
    a = torch.exp(log_a)
    S, out = u.new_zeros(width), torch.zeros_like(u)
    for t in range(n):
        S = a[t] * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(h, W, p, m, eps, dt):
    g = lambda name: W[p + name].to(dt)
    y = gelu_tanh(h @ g("y").T + g("y.b"))
    u = causal_conv(h @ g("x").T + g("x.b"), g("conv"), g("conv.b"))
    return (linear_recurrence(u, W, p, m, dt) * y) @ g("o").T


def side_by_side(h, W, p, m, eps, dt):
    left = rms(window_attention(h, W, p + "left.", m["left"], eps, dt), eps) * W[p + "left.out"].to(dt)
    right = rms(recurrent_block(h, W, p + "right.", m["right"], eps, dt), eps) * W[p + "right.out"].to(dt)
    return 0.5 * (left + right)


MIXERS = {"gla": gla, "lightning": lightning, "parallel": side_by_side}


# ---------------------------------------------------------------- feed-forwards
def gated_ff(h, W, p, act, dt):
    g = lambda name: W[p + name].to(dt)
    return (act(h @ g("gate").T) * (h @ g("up").T)) @ g("down").T


def route(h, W, p, top, dt):
    """(chosen experts [n, top], weights [n, top], margin [n]: how far the last chosen logit lies above the best one left out)."""
    z = h @ W[p + "router"].to(dt).T
    vals, idx = torch.topk(z, top, dim=-1)
    if top < z.shape[-1]:
        margin = vals[:, -1] - torch.topk(z, top + 1, dim=-1).values[:, -1]
    else:
        margin = torch.full((z.shape[0],), float("inf"), dtype=dt)
    return idx, torch.softmax(vals, dim=-1), margin


def moe_ff(h, W, p, mlp, dt, margins=None):
    top = int(mlp["router"]["top"])
    idx, w, margin = route(h, W, p, top, dt)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        share = (w * (idx == e)).sum(-1, keepdim=True)
        used = share[:, 0] > 0
        if used.any():
            out[used] = out[used] + share[used] * gated_ff(h[used], W, f"{p}e{e}.", silu, dt)
    if mlp.get("shared"):
        out = out + gated_ff(h, W, p + "shared.", silu, dt)
    return out


# ---------------------------------------------------------------- the model
def forward(cfg, W, tokens, dt=torch.float64, layers_out=None, margins=None, noise=None):
    """Logits [n, vocab] of one whole sequence; `layers_out` (a list) receives the stream after every layer, `margins` (a
    list) every router's margins [n]; `noise` (a function) is applied to what the sublayers read and return (rounding to 16
    bits there shows how far a row moves under it)."""
    noise = noise or (lambda t: t)
    eps = float(cfg["norm"]["eps"])
    norm = lambda x, name: rms(x, eps) * (1.0 + W[name].to(dt))
    x = embedded(cfg, W, tokens, dt)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = token_shift(noise(norm(x, p + "norm1")), W[p + "shift"].to(dt))
        y = noise(MIXERS[layer["type"]](noise(h), W, p + "mix.", layer["mixer"], eps, dt))
        x = x + norm(y, p + "norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = noise(norm(x, p + "norm2"))
            y = gated_ff(h, W, p + "mlp.", gelu_tanh, dt) if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp, dt, margins)
            x = x + norm(noise(y), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ W["head"].to(dt).T
