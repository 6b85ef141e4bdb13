"""A plain, slow restatement of the Gonozen design in 64-bit torch: whole sequences, no cache, no kernels.

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


def rms_norm(x, weight, eps):
    return _d(x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight)


def frequencies(rot):
    """(angle per position of each pair, factor of cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def place(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    first = max(math.floor(place(sc["fast"])), 0)
    last = min(math.ceil(place(sc["slow"])), dims - 1)
    share = ((i - first) / max(last - first, 0.001)).clamp(0.0, 1.0)
    return f / sc["factor"] * share + f * (1 - share), 0.1 * math.log(sc["factor"]) + 1.0


def turn(x, positions, rot):
    """x [T, ..., n]: entries i and i + dims/2 of the last axis turn by p * f_i; entries behind dims stay."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f, amplitude = frequencies(rot)
    angle = positions.to(F64)[:, None] * f[None, :]
    angle = angle.reshape(angle.shape[:1] + (1,) * (x.dim() - 2) + angle.shape[1:])
    c, s = amplitude * torch.cos(angle), amplitude * torch.sin(angle)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def visible(T, window=None):
    """[T, T]: entry [i, j] is true when position i sees j (window None: every j <= i; else the last `window` of them)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < (T if window is None else window))


def weights_of_scores(scores, sees, sinks=None):
    """Softmax over the visible keys of scores [heads, T, T]; `sinks` [heads]: one more term exp(sink) in the denominator."""
    s = scores.masked_fill(~sees, -math.inf)
    top = s.amax(dim=-1, keepdim=True)
    if sinks is not None:
        top = torch.maximum(top, sinks[:, None, None].expand_as(top))
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if sinks is not None:
        total = total + torch.exp(sinks[:, None, None] - top)
    return e / total


def latent_attention(h, w, p, m, positions, eps, weights_out=None):
    """A rotated key part for all heads beside keys made from the latent; a sigmoid gate per head on the output."""
    T, H, d, r, vd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(h, w[p + "q"]).view(T, H, d + r)
    down = lin(h, w[p + "dkv"])
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    q_rot, k_rot = _d(turn(q[..., d:], positions, m.get("rot"))), _d(turn(down[:, rank:], positions, m.get("rot")))
    k = lin(c, w[p + "uk"]).view(T, H, d)
    v = lin(c, w[p + "uv"]).view(T, H, vd)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    pr = weights_of_scores(scores, visible(T))
    if weights_out is not None:
        weights_out.append(pr)
    o = _d(torch.einsum("hij,jhd->ihd", pr, v)) * torch.sigmoid(lin(h, w[p + "g"]))[:, :, None]
    return lin(o.reshape(T, H * vd), w[p + "o"])


def latent_attention_2(h, w, p, m, eps, weights_out=None):
    """Queries through a latent of their own, no positions, a sliding window, a sink per head."""
    T, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = lin(rms_norm(lin(h, w[p + "dq"]), w[p + "dq.norm"], eps), w[p + "uq"]).view(T, H, d)
    c = rms_norm(lin(h, w[p + "dkv"]), w[p + "dkv.norm"], eps)
    k = lin(c, w[p + "uk"]).view(T, H, d)
    v = lin(c, w[p + "uv"]).view(T, H, vd)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    pr = weights_of_scores(scores, visible(T, (m.get("mask") or {}).get("size")), w[p + "sink"])
    if weights_out is not None:
        weights_out.append(pr)
    o = _d(torch.einsum("hij,jhd->ihd", pr, v))
    return lin(o.reshape(T, H * vd), w[p + "o"])


def expert(h, w, p, limit):
    g, u = lin(h, w[p + "gate"]), lin(h, w[p + "up"])
    if limit is not None:
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return lin(_d(g * torch.sigmoid(1.702 * g) * (u + 1)), w[p + "down"])


def route(z, top, groups=None, margins=None):
    """z [T, E] router sums. (chosen experts [T, top] by descending score, their weights [T, top]). `margins`: a list that
    gets, per row, the smallest distance of a score that decided something from one that would have decided otherwise, as a
    difference of logarithms (the smaller of the groups' and the experts')."""
    T, E = z.shape
    s = torch.softmax(z, dim=-1)
    c, tight = s, torch.full((T,), math.inf, dtype=F64)
    if groups and groups["count"] > 1:
        n, keep = groups["count"], groups["keep"]
        best = s.view(T, n, E // n).amax(dim=-1)
        val, order = torch.sort(best, dim=-1, descending=True, stable=True)
        if keep < n:
            tight = torch.log(val[:, keep - 1]) - torch.log(val[:, keep])
        kept = torch.zeros(T, n, dtype=torch.bool).scatter_(1, order[:, :keep], True)
        c = s.masked_fill(~kept.repeat_interleave(E // n, dim=1), -math.inf)
    val, order = torch.sort(c, dim=-1, descending=True, stable=True)
    if top < E:
        nxt = val[:, top]
        tight = torch.where(nxt > 0, torch.minimum(tight, torch.log(val[:, top - 1]) - torch.log(nxt.clamp_min(1e-300))), tight)
    if margins is not None:
        margins.append(tight)
    picked = val[:, :top]
    return order[:, :top], picked / (picked.sum(dim=-1, keepdim=True) + 1e-20)


def mixture(h, w, p, m, margins=None):
    r = m["router"]
    idx, wt = route(h @ w[p + "router"].T, r["top"], r.get("groups"), margins)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        hit = idx == e
        rows = hit.any(dim=1)
        if rows.any():
            out[rows] += (wt * hit).sum(dim=1)[rows, None] * expert(h[rows], w, f"{p}e{e}.", m["expert"].get("limit"))
    if m.get("shared"):
        out = out + expert(h, w, p + "shared.", m["shared"].get("limit"))
    return out


def forward(tokens, cfg, w, layers_out=None, margins=None):
    """`margins`: a list that gets, per mixture, how clear each row's choice of experts is (see `route`)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens]
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if L["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, positions, eps)
        elif L["type"] == "latent_attention_2":
            y = latent_attention_2(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(L["type"])
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            x = x + rms_norm(mixture(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"], margins), w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    z = lin(rms_norm(x, w["final.norm"], eps), w["embed"])
    cap = cfg.get("logit_softcap")
    return z if not cap else cap * torch.tanh(z / cap)
