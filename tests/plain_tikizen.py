"""A plain, slow restatement of the Tikizen design in 64-bit torch: whole sequences, no cache, no kernels.

One function per mechanism; nothing here is shared with the product path. `cfg` is the design's config.json as a
dictionary, `w` maps tensor names to 64-bit tensors. `forward` returns the logits of every position and, if asked,
the stream after every layer."""
from __future__ import annotations

import math

import torch

F64 = torch.float64

# Inside `disturbed(rel, seed)` every product and every norm is multiplied by 1 + rel * u, u uniform in [-1, 1) and drawn
# anew for every entry, which is what a 16-bit engine's roundings do; the difference from the exact run measures, row by
# row, what rounding alone causes.
_NOISE = []


class disturbed:
    def __init__(self, rel, seed):
        self.rel, self.gen = rel, torch.Generator().manual_seed(seed)

    def __enter__(self):
        _NOISE.append(self)

    def __exit__(self, *a):
        _NOISE.pop()


def _d(x):
    if not _NOISE:
        return x
    n = _NOISE[-1]
    return x * (1 + n.rel * (2 * torch.rand(x.shape, generator=n.gen, dtype=F64) - 1))


def lin(h, W):
    return _d(h @ W.T)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def rms(x, eps):
    return _d(x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps))


def frequencies(rot):
    """(angle per position of each pair, factor of cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    half = dims // 2
    i = torch.arange(half, dtype=F64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    at = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(at(sc["fast"])), 0)
    hi = min(math.ceil(at(sc["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_half(x, positions, rot):
    """x [T, heads, d]: entries i and i + dims/2 of every head turn by p * f_i; the rest stay."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    half = dims // 2
    f, amp = frequencies(rot)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = (amp * torch.cos(ang))[:, None, :], (amp * torch.sin(ang))[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T, chunk=None):
    """[T, T] mask: entry [i, j] is true when j <= i and both lie in one chunk (chunk None: every earlier key)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    if chunk is not None:
        m = m & (i // chunk == j // chunk)
    return m


def attention(h, w, p, m, positions, eps, kept=None, weights_out=None):
    """Attention with unit-RMS rotated queries and keys inside chunks. `kept`: the (keys, values) of another layer, which
    are read instead of own ones. Returns (result, (keys, values))."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, vd = m.get("kv_heads", H), m.get("vdim", d)
    rot = m.get("rot")
    q = rms(rotate_half(lin(h, w[p + "q"]).view(T, H, d), positions, rot), eps)
    if kept is None:
        k = rms(rotate_half(lin(h, w[p + "k"]).view(T, G, d), positions, rot), eps)
        kept = (k, lin(h, w[p + "v"]).view(T, G, vd))
    k, v = kept
    kk, vv = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * m["scale"]
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size"))[None], -math.inf)
    pr = torch.softmax(s, dim=-1)
    if weights_out is not None:
        weights_out.append(pr)
    o = _d(torch.einsum("hij,jhd->ihd", pr, vv))
    return lin(o.reshape(T, H * vd), w[p + "o"]), kept


def decayed_sums(q, k, v, decay, write):
    """S <- decay S + write k v^T;  o = S^T q. q, k [T, heads, N], v [T, heads, vd], decay and write [T, heads]."""
    T, H, N = q.shape
    S = torch.zeros(H, N, v.shape[2], dtype=F64)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + (write[t][:, None] * k[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnj,hn->hj", S, q[t]))
    return torch.stack(out)


def retention(h, w, p, m, positions, eps):
    T = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot")
    q = rotate_half(lin(h, w[p + "q"]).view(T, H, d), positions, rot)
    k = rotate_half(lin(h, w[p + "k"]).view(T, H, d), positions, rot) * d ** -0.5
    v = lin(h, w[p + "v"]).view(T, H, vd)
    decay = torch.tensor(m["decay"], dtype=F64)[None].expand(T, H)
    o = rms(decayed_sums(q, k, v, decay, torch.ones(T, H, dtype=F64)), eps)
    return lin(o.reshape(T, H * vd) * silu(lin(h, w[p + "g"])), w[p + "o"])


def causal_conv(u, taps, bias):
    """u [T, C], taps [C, n]: the last column weighs the current row; zeros before the start."""
    T, n = u.shape[0], taps.shape[1]
    past = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=F64), u])
    return sum(past[j:j + T] * taps[:, j] for j in range(n)) + bias


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, vd, N, G, ng = m["heads"], m["vdim"], m["state"], m.get("groups", 1), m.get("norm_groups", 1)
    inner = H * vd
    z, x, B, C, dt = torch.split(lin(h, w[p + "in"]), [inner, inner, G * N, G * N, H], dim=1)
    xBC = silu(causal_conv(torch.cat([x, B, C], dim=1), w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(_d(xBC), [inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[p + "dt_bias"])
    x = x.view(T, H, vd)
    B = B.view(T, G, N).repeat_interleave(H // G, dim=1)
    C = C.view(T, G, N).repeat_interleave(H // G, dim=1)
    y = decayed_sums(C, B, x, torch.exp(-torch.exp(w[p + "A_log"]) * dt), dt) + w[p + "D"][None, :, None] * x
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, ng, inner // ng), eps).reshape(T, inner) * w[p + "norm"]
    return lin(y, w[p + "o"])


def dense(h, w, p, limit):
    g, u = lin(h, w[p + "gate"]), lin(h, w[p + "up"])
    if limit is not None:
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return lin(_d(g * torch.sigmoid(1.702 * g) * (u + 1)), w[p + "down"])


def expert(h, w, p):
    return lin(_d(silu(lin(h, w[p + "gate"])) * lin(h, w[p + "up"])), w[p + "down"])


def choose(z, top):
    """(indices of the `top` largest of each row, the softmax over them)."""
    val, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    return idx[:, :top], torch.softmax(val[:, :top], dim=-1)


def mixture(h, w, p, m, margins=None):
    z = h @ w[p + "router"].T + w[p + "router.b"]
    top = m["router"]["top"]
    idx, wt = choose(z, top)
    if margins is not None and top < z.shape[1]:
        s = torch.sort(z, dim=-1, descending=True).values
        margins.append(s[:, top - 1] - s[:, top])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        hit = (idx == e)
        rows = hit.any(dim=1)
        if rows.any():
            out[rows] += (wt * hit).sum(dim=1)[rows, None] * expert(h[rows], w, f"{p}e{e}.")
    if m.get("shared"):
        out = out + torch.sigmoid(lin(h, w[p + "shared.sg"])) * expert(h, w, p + "shared.")
    return out


def feed_forward(x, w, p, m, margins=None):
    return dense(x, w, p, m.get("limit")) if m["kind"] == "dense" else mixture(x, w, p, m, margins)


def forward(tokens, cfg, w, layers_out=None, margins=None):
    """`margins`: a list that gets, per mixture, how far each row's last chosen logit lies above the first left out."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    eps, alpha = cfg["norm"]["eps"], cfg.get("postln_alpha", 1.0)
    x = rms(w["embed"][tokens], eps) * w["embed.norm"]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "retention":
            y = retention(x, w, p + "mix.", m, positions, eps)
        elif L["type"] == "mamba2":
            y = mamba2(x, w, p + "mix.", m, eps)
        elif L["type"] == "attention":
            y, kept[i] = attention(x, w, p + "mix.", m, positions, eps, kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            raise ValueError(L["type"])
        x = rms(alpha * x + y, eps) * w[p + "norm1"]
        if L.get("mlp") is not None:
            x = rms(alpha * x + feed_forward(x, w, p + "mlp.", L["mlp"], margins), eps) * w[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x)
    return lin(rms(x, eps) * w["final.norm"], w["head"])
