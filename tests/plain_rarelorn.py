"""The Rarelorn decoder, plainly: float64 torch on the CPU, one function per mechanism, whole sequences at once (no
cache, no batching, no portions; recurrences walk the tokens one by one).  It shares nothing with the library; the tests
compare the library with it.

A sequence's positions are 0 .. n-1.  `w` maps tensor names to float tensors, `c` is the configuration as the
model's config.json gives it."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def scalar_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """An RMS norm with one gain for all channels."""
    return unit_rms(x, eps) * gain.reshape(())


def short_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [n, channels], taps [channels, J]: y_t = sum_j taps[:, j] u_(t - J + 1 + j), nought before the first token."""
    n, J = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(J - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + n] * taps[:, j] for j in range(J))


def rotate_halves(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [n, heads, d]: channel i < dims/2 of every head is paired with channel i + dims/2; the rest pass."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    half = dims // 2
    f = rot["base"] ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    angle = torch.arange(x.shape[0], dtype=F64)[:, None] * f[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., dims:]], dim=-1)


def visible(n: int, window: Optional[int]) -> torch.Tensor:
    """[query, key]: key j is seen from position i when 0 <= i - j (< window)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    if window:
        see = see & (i - j < window)
    return see


def sigmoid_weights(scores: torch.Tensor, see: torch.Tensor, temp, cap: Optional[float], bias) -> torch.Tensor:
    """Weights of the keys, each by itself: sigmoid(cap tanh(temp score / cap) + bias) where seen, else nought."""
    s = scores * temp
    if cap:
        s = cap * torch.tanh(s / cap)
    return torch.sigmoid(s + bias) * see


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    """Sigmoid attention with a short convolution on q, k and v."""
    n = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    q, k, v = (h @ w[p + x].T + w[p + x + ".b"] for x in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(u, w[p + x + ".conv"]) for x, u in zip("qkv", (q, k, v)))
    q = rotate_halves(q.view(n, H, d), m.get("rot"))
    k = rotate_halves(k.view(n, G, d), m.get("rot"))
    v = v.view(n, G, dv)
    see = visible(n, (m.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        weights = sigmoid_weights((q[:, a] @ k[:, g].T) * m["scale"], see, w[p + "temp"][a], m.get("softcap"), w[p + "pb"][a])
        heads.append(weights @ v[:, g])
    return torch.cat(heads, dim=-1) @ w[p + "o"].T + w[p + "o.b"]


def previous(h: torch.Tensor) -> torch.Tensor:
    """Every token's predecessor, nought before the first."""
    return torch.cat([torch.zeros(1, h.shape[1], dtype=h.dtype), h[:-1]])


def bonus_recurrence(r, k, v, w, u):
    """r, k, w [n, H, d], v [n, H, dv], u [H, d]: o_t = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    n, H, d = k.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64)
    out = []
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t]))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out)


def time_mixing(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    n, H, d = h.shape[0], m["heads"], m["dim"]
    before = previous(h)
    mixed = {x: h + (before - h) * w[p + "mu." + x] for x in "rkvgw"}
    r, k, v = ((mixed[x] @ w[p + x].T).view(n, H, d) for x in "rkv")
    gate = silu(mixed["g"] @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(n, H, d)
    o = unit_rms(bonus_recurrence(r, k, v, decay, w[p + "u"]), eps).reshape(n, H * d)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return m["left_scale"] * attention(h, w, p + "left.", m["left"]) + m["right_scale"] * time_mixing(h, w, p + "right.", m["right"], eps)


def matrix_memory(q, k, v, i, f):
    """q, k [n, H, d], v [n, H, dv], log gates i, f [n, H]: the stabilised matrix memory, its maximum starting at 0."""
    n, H, d = k.shape
    S, N, top = torch.zeros(H, d, v.shape[-1], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    out = []
    for t in range(n):
        new = torch.maximum(f[t] + top, i[t])
        keep, learn = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        top = new
        S = keep[:, None, None] * S + learn[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        N = keep[:, None] * N + learn[:, None] * k[t]
        den = torch.maximum((N * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hij,hi->hj", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    n, H, d = h.shape[0], m["heads"], m["dim"]
    dv, cap = m.get("vdim", d), m["gate_cap"]
    q = (h @ w[p + "q"].T).view(n, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(n, H, d)
    v = (h @ w[p + "v"].T).view(n, H, dv)
    capped = lambda x: cap * torch.tanh((h @ w[p + x].T + w[p + x + ".b"]) / cap)
    o = matrix_memory(q, k, v, capped("i"), torch.nn.functional.logsigmoid(capped("f")))
    o = unit_rms(o, eps).reshape(n, H * dv) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_recurrence(q, k, v, g, beta):
    """q, k [n, H, d], v [n, H, dv], g, beta [n, H]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    n, H, d = k.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64)
    out = []
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hij,hi->hj", S, q[t]))
    return torch.stack(out)


def delta(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    n, H, d = h.shape[0], m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    q, k, v = (h @ w[p + x].T for x in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(u, w[p + x + ".conv"]) for x, u in zip("qkv", (q, k, v)))
    q, k, v = silu(q).view(n, G, d), silu(k).view(n, G, d), silu(v).view(n, H, dv)
    unit = lambda x: x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q) * d ** -0.5, unit(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * torch.nn.functional.softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = unit_rms(delta_recurrence(q, k, v, g, beta), eps) * w[p + "norm"]
    return (o.reshape(n, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, r: dict):
    """-> chosen [n, top] (indices), weights [n, top], margin [n]: how far the last chosen logit lies above the best one
    left out, among experts and among groups (a small margin is a close call that rounding may turn)."""
    E, top = r["experts"], r["top"]
    z = h @ w[p + "router"].T
    s = torch.softmax(z, -1)
    choice = z                                                      # softmax keeps the order
    margin = torch.full((h.shape[0],), float("inf"), dtype=F64)
    groups = r.get("groups")
    if groups:
        by_group = choice.view(-1, groups["count"], E // groups["count"])
        score = by_group.max(-1).values
        ranked = score.sort(dim=-1, descending=True)
        kept = torch.zeros_like(score, dtype=torch.bool)
        kept.scatter_(1, ranked.indices[:, :groups["keep"]], True)
        choice = by_group.masked_fill(~kept[:, :, None], -float("inf")).reshape(-1, E)
        if groups["keep"] < groups["count"]:
            margin = ranked.values[:, groups["keep"] - 1] - ranked.values[:, groups["keep"]]
    ranked = choice.sort(dim=-1, descending=True)
    chosen = ranked.indices[:, :top]
    if top < E:
        margin = torch.minimum(margin, ranked.values[:, top - 1] - ranked.values[:, top])
    return chosen, s.gather(1, chosen) * r.get("scale", 1.0), margin


def experts(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, f: dict, margins: Optional[list] = None) -> torch.Tensor:
    chosen, weights, margin = route(h, w, p, f["router"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in chosen.unique().tolist():
        rows, place = (chosen == e).nonzero(as_tuple=True)
        out[rows] += weights[rows, place, None] * gated_unit(h[rows], w, f"{p}e{e}.")
    return out


def order_of_runs(c: dict) -> List[tuple]:
    """(layer, pass): pass t at the first layer of the loop's t-th pass, else None."""
    n, loop = len(c["layers"]), c.get("loop")
    if not loop or loop["start"] == loop["stop"]:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop.get("times", 1)):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(c: dict, w: Dict[str, torch.Tensor], tokens: List[int], after_runs: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab].  `after_runs` receives the stream after every layer run, `margins` the routers' margins."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = c["norm"]["eps"]
    x0 = w["embed"][torch.tensor(tokens)]
    x = x0
    for i, t in order_of_runs(c):
        if t is not None:
            x = (x + x0 if t > 0 else x) + w["loop.step"][t]
        L, p = c["layers"][i], f"l{i}."
        m, h = L["mixer"], scalar_norm(x, w[p + "norm1"], eps)
        if L["type"] == "delta":
            x = x + delta(h, w, p + "mix.", m, eps)
        elif L["type"] == "mlstm":
            x = x + mlstm(h, w, p + "mix.", m, eps)
        else:
            x = x + side_by_side(h, w, p + "mix.", m, eps)
        if L.get("mlp") is not None:
            x = x + experts(scalar_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"], margins)
        if after_runs is not None:
            after_runs.append(x)
    return scalar_norm(x, w["final.norm"], eps) @ w["head"].T
