"""Plain, slow Nesezen forward pass: whole sequences, no cache, one function per mechanism.

The oracle for the engine's Nesezen model.  It shares no code with the package: it reads a model folder with its own
few lines (or takes a dict of tensors), works on one whole sequence at a time and keeps nothing between calls.  Every
function works in the dtype `dt` it is given (float64 for an oracle); nothing is rounded below `dt`.

Notation: n tokens, D the model width.  A layer is

    x += mixer(N1(x));   x += ff(N2(x)),          N(x) = tanh(alpha x) * w + b

N computes no statistics of its row.  The mixer is `attention` (windowed, partly rotated heads, capped scores), `mlstm`
(a matrix state per head with exponential gates held in range by a running maximum) or `latent_attention` (low-rank
queries, keys and values without positions, a gate a head).  The feed-forward is a gated SiLU layer, a mixture of such
layers whose weights multiply the experts' INPUTS, beside a shared one with a gate of its own, or absent.
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


def log_sigmoid(x):
    return torch.minimum(x, torch.zeros_like(x)) - torch.log1p(torch.exp(-x.abs()))


def tanh_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


# ---------------------------------------------------------------- windowed attention with capped scores
def stretched_frequencies(dims, base, scaling):
    """f_i of pair i (i < dims / 2): waves longer than `original / low` are slowed by `factor`, shorter than
    `original / high` kept, and between the two the frequency goes linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_front_halves(x, rot, dt):
    """x [n, heads, dim]: among the first rot.dims elements, i turns with i + dims/2; the rest stays."""
    dims = int(rot["dims"]) if rot else 0
    if dims == 0:
        return x
    half = dims // 2
    freq = stretched_frequencies(dims, float(rot["base"]), rot.get("scaling")).to(dt)
    ang = torch.arange(x.shape[0], dtype=dt)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def capped(scores, cap):
    return cap * torch.tanh(scores / cap) if cap else scores


def visible(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i - j < size) if size else (j <= i)


def attention(h, W, p, m, eps, dt):
    n = h.shape[0]
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda name: W[p + name].to(dt)
    q = rotate_front_halves((h @ g("q").T).reshape(n, H, dk), m.get("rot"), dt)
    k = rotate_front_halves((h @ g("k").T).reshape(n, G, dk), m.get("rot"), dt)
    v = (h @ g("v").T).reshape(n, G, dv)
    kh = torch.arange(H) // (H // G)
    s = capped(torch.einsum("ihd,jhd->hij", q, k[:, kh]) * float(m["scale"]), float(m.get("softcap") or 0.0))
    s = s.masked_fill(~visible(n, int((m.get("mask") or {}).get("size") or 0)), float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v[:, kh]).reshape(n, H * dv) @ g("o").T


# ---------------------------------------------------------------- matrix memory with exponential gates
def mlstm_gates(zi, zf, cap):
    """Log gates of the pre-activations: the input gate soft-capped, the forget gate log sigmoid of the soft-capped."""
    return cap * torch.tanh(zi / cap), log_sigmoid(cap * torch.tanh(zf / cap))


def mlstm_recurrence(q, k, v, i, f):
    """q, k [n, H, dk], v [n, H, dv], log gates i, f [n, H]: o [n, H, dv], from a state of zeros (the running maximum, too,
    starts at 0)."""
    n, H, dk = q.shape
    m, maxima = q.new_zeros(H), []
    for t in range(n):
        m = torch.maximum(f[t] + m, i[t])
        maxima.append(m)
    m = torch.stack(maxima)
    before = torch.cat([torch.zeros_like(m[:1]), m[:-1]])
    keep, put = torch.exp(f + before - m), torch.exp(i - m)
    # the normaliser is one more value column that holds ones
    S, w, v1 = q.new_zeros((H, dk, v.shape[2] + 1)), put[:, :, None] * k, torch.cat([v, torch.ones_like(v[:, :, :1])], dim=-1)
    out = []
    for t in range(n):
        S = keep[t][:, None, None] * S + w[t][:, :, None] * v1[t][:, None, :]
        out.append((q[t][:, None, :] @ S)[:, 0])
    out = torch.stack(out)
    floor = torch.maximum(out[..., -1].abs(), torch.exp(-m))
    return out[..., :-1] / (floor + 1e-6)[..., None]


def mlstm(h, W, p, m, eps, dt, noise=None):
    """`noise` (a function) is applied to the projections."""
    n = h.shape[0]
    H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda name: W[p + name].to(dt)
    made = lambda name: (noise or (lambda t: t))(h @ g(name).T)
    q, k, v = made("q").reshape(n, H, dk) * dk ** -0.5, made("k").reshape(n, H, dk), made("v").reshape(n, H, dv)
    i, f = mlstm_gates(made("i") + g("i.b"), made("f") + g("f.b"), float(m["gate_cap"]))
    o = rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(n, H * dv)
    return (o * g("norm") * sigmoid(made("g"))) @ g("o").T


# ---------------------------------------------------------------- attention through a latent, without positions
def latent_attention(h, W, p, m, eps, dt):
    n = h.shape[0]
    H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda name: W[p + name].to(dt)
    q = ((rms(h @ g("dq").T, eps) * g("dq.norm")) @ g("uq").T).reshape(n, H, dk)
    c = rms(h @ g("dkv").T, eps) * g("dkv.norm")
    k, v = (c @ g("uk").T).reshape(n, H, dk), (c @ g("uv").T).reshape(n, H, dv)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    s = s.masked_fill(~visible(n, 0), float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v)
    o = o * sigmoid(h @ g("g").T)[:, :, None]
    return o.reshape(n, H * dv) @ g("o").T


MIXERS = {"attention": attention, "mlstm": mlstm, "latent_attention": latent_attention}


# ---------------------------------------------------------------- feed-forwards
def gated_ff(h, W, p, dt):
    g = lambda name: W[p + name].to(dt)
    return (silu(h @ g("gate").T) * (h @ g("up").T)) @ g("down").T


def route(h, W, p, top, dt):
    """(chosen experts [n, top], weights [n, top], margin [n]: how far the last chosen logit lies above the best one left out)."""
    z = h @ W[p + "router"].to(dt).T
    vals, idx = torch.topk(z, top, dim=-1)
    if top < z.shape[-1]:
        margin = vals[:, -1] - torch.topk(z, top + 1, dim=-1).values[:, -1]
    else:
        margin = torch.full((z.shape[0],), float("inf"), dtype=dt)
    return idx, sigmoid(vals), margin


def moe_ff(h, W, p, mlp, dt, margins=None):
    """The sum of expert(w * h) over the chosen experts, and the shared expert times its own gate."""
    idx, w, margin = route(h, W, p, int(mlp["router"]["top"]), dt)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        chosen = idx == e
        used = chosen.any(-1)
        if used.any():
            share = (w * chosen).sum(-1, keepdim=True)[used]
            out[used] = out[used] + gated_ff(share * h[used], W, f"{p}e{e}.", dt)
    if mlp.get("shared"):
        out = out + gated_ff(h, W, p + "shared.", dt) * sigmoid(h @ W[p + "shared.sg"].to(dt).T)
    return out


# ---------------------------------------------------------------- the model
def forward(cfg, W, tokens, dt=torch.float64, layers_out=None, margins=None, noise=None):
    """Logits [n, vocab] of one whole sequence; `layers_out` (a list) receives the stream after every layer, `margins` (a
    list) every router's margins [n]; `noise` (a function) is applied to what the sublayers read and return (rounding to 16
    bits there shows how far a row moves under it)."""
    noise = noise or (lambda t: t)
    eps = float(cfg["norm"]["eps"])
    norm = lambda x, name: tanh_norm(x, W[name + ".alpha"].to(dt).reshape(()), W[name].to(dt), W[name + ".b"].to(dt))
    x = W["embed"].to(dt)[torch.as_tensor(list(tokens), dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = int(cfg["layers"][j]["weights_of"])
        p, mlp = f"l{j}.", layer.get("mlp")
        x = x + noise(MIXERS[layer["type"]](noise(norm(x, p + "norm1")), W, p + "mix.", layer["mixer"], eps, dt))
        if mlp is not None:
            h = noise(norm(x, p + "norm2"))
            y = gated_ff(h, W, p + "mlp.", dt) if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp, dt, margins)
            x = x + noise(y)
        if layers_out is not None:
            layers_out.append(x.clone())
    return noise(norm(x, "final.norm")) @ W["head"].to(dt).T
