"""The Fomodra decoder, plainly: float64 torch on the CPU, one function per mechanism, whole sequences at once (no
cache, no batching, no portions; the recurrence walks the tokens one by one).  It shares nothing with the library; the tests
compare the library with it.

A sequence's positions are 0 .. n-1.  `w` maps tensor names to float tensors, `c` is the configuration as the
model's config.json gives it."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64
SIGMOID_SLOPE = 1.702


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * weight


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_rows(c: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """A token's row plus the row of the pair (token before, token); a sequence's first token takes the pairs' last row."""
    x = w["embed"][torch.tensor(tokens)]
    pair = (c.get("embedding") or {}).get("bigram")
    if pair:
        rows = [pair["buckets"]] + [(a * pair["mul_prev"] + b * pair["mul_cur"]) % pair["buckets"] for a, b in zip(tokens, tokens[1:])]
        x = x + w["bigram"][torch.tensor(rows)]
    return x


def frequencies(rot: dict) -> torch.Tensor:
    """The angular frequency of every pair; with scaling, long wavelengths are stretched, short ones kept."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            length = 2.0 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_halves(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [n, heads, d]: channel i < dims/2 of every head is paired with channel i + dims/2; the rest pass."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    half = dims // 2
    angle = torch.arange(x.shape[0], dtype=F64)[:, None] * frequencies(rot)[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., dims:]], dim=-1)


def visible(n: int, window: Optional[int] = None, chunk: Optional[int] = None) -> torch.Tensor:
    """[query, key]: key j <= i is seen from position i when i - j < window, or when both lie in the same chunk."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    if window:
        see = see & (i - j < window)
    if chunk:
        see = see & (i // chunk == j // chunk)
    return see


def softmax_with_sink(scores: torch.Tensor, see: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the seen keys; with `sink` the denominator also holds exp(sink), which belongs to no key."""
    s = scores.masked_fill(~see, -float("inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    denom = e.sum(-1, keepdim=True)
    if sink is not None:
        denom = denom + torch.exp(sink - top)
    return e / denom


def grouped_heads(q, k, v, see, scale, sinks=None) -> torch.Tensor:
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> the heads' results one beside the other, [n, H * dv]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for a in range(H):
        g = a // (H // G)
        prob = softmax_with_sink((q[:, a] @ k[:, g].T) * scale, see, None if sinks is None else sinks[a])
        out.append(prob @ v[:, g])
    return torch.cat(out, dim=-1)


def mask_size(m: dict) -> Optional[int]:
    return (m.get("mask") or {}).get("size")


def windowed_attention(h, w, p, m, kept: Dict[int, tuple], layer: int) -> torch.Tensor:
    """Biases, a rotation, a window, a sink per head.  `kept` holds every layer's rotated keys and values; a layer with
    `kv_from` takes those of the layer it names."""
    n = h.shape[0]
    H, G, d = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    q = rotate_halves((h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d), m.get("rot"))
    if m.get("kv_from") is not None:
        k, v = kept[m["kv_from"]]
    else:
        k = rotate_halves((h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d), m.get("rot"))
        v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, m.get("vdim", d))
        kept[layer] = (k, v)
    heads = grouped_heads(q, k, v, visible(n, window=mask_size(m)), m["scale"], w[p + "sink"])
    return heads @ w[p + "o"].T


def chunked_attention(h, w, p, m) -> torch.Tensor:
    n = h.shape[0]
    H, G, d = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    q = rotate_halves((h @ w[p + "q"].T).view(n, H, d), m.get("rot"))
    k = rotate_halves((h @ w[p + "k"].T).view(n, G, d), m.get("rot"))
    v = (h @ w[p + "v"].T).view(n, G, m.get("vdim", d))
    return grouped_heads(q, k, v, visible(n, chunk=mask_size(m)), m["scale"]) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps) -> torch.Tensor:
    n = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m.get("vdim", m["dim"]), m["kv_rank"]
    q = (h @ w[p + "q"].T).view(n, H, d + r)
    down = h @ w[p + "dkv"].T
    lat = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    shared = rotate_halves(down[:, None, R:], m.get("rot"))[:, 0]
    q_plain, q_rot = q[..., :d], rotate_halves(q[..., d:], m.get("rot"))
    k_plain = (lat @ w[p + "uk"].T).view(n, H, d)
    v = (lat @ w[p + "uv"].T).view(n, H, dv)
    see = visible(n, window=mask_size(m))
    gate = torch.sigmoid(h @ w[p + "g"].T)
    heads = []
    for a in range(H):
        scores = (q_plain[:, a] @ k_plain[:, a].T + q_rot[:, a] @ shared.T) * m["scale"]
        heads.append(softmax_with_sink(scores, see, w[p + "sink"][a]) @ v[:, a] * gate[:, a:a + 1])
    return torch.cat(heads, dim=-1) @ w[p + "o"].T


def short_conv(u: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [n, channels], taps [channels, J]: y_t = bias + sum_j taps[:, j] u_(t - J + 1 + j), nought before the first token."""
    n, J = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(J - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + n] * taps[:, j] for j in range(J)) + bias


def selective_scan(x, dt, A, B, C, D) -> torch.Tensor:
    """x, dt [n, channels], A [channels, N], B, C [n, N]: S <- exp(dt A) S + dt x B, y = S C + D x, S nought at first."""
    S = torch.zeros_like(A)
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out)


def selective_mixer(h, w, p, m) -> torch.Tensor:
    inner, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(short_conv(x, w[p + "conv"], w[p + "conv.b"]))
    low = x @ w[p + "x"].T
    dt = torch.nn.functional.softplus(low[:, :R] @ w[p + "dt"].T + w[p + "dt.b"], threshold=1e9)
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), low[:, R:R + N], low[:, R + N:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def two_mixers(h, w, p, m, eps) -> torch.Tensor:
    left = rms_norm(chunked_attention(h, w, p + "left.", m["left"]), w[p + "left.out"], eps)
    right = rms_norm(selective_mixer(h, w, p + "right.", m["right"]), w[p + "right.out"], eps)
    return 0.5 * (left + right)


def bounded_unit(h, w, p, limit) -> torch.Tensor:
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(SIGMOID_SLOPE * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, w, p, r):
    """-> chosen [n, top] (indices), weights [n, top], margin [n]: how far the last chosen corrected score lies above
    the best one left out (a small margin is a close call that rounding may turn)."""
    total, top = r["experts"] + r.get("identity", 0), r["top"]
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    ranked = (s + w[p + "correction"]).sort(dim=-1, descending=True)
    chosen = ranked.indices[:, :top]
    margin = ranked.values[:, top - 1] - ranked.values[:, top] if top < total else torch.full((h.shape[0],), float("inf"), dtype=F64)
    picked = s.gather(1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20), margin


def experts(h, w, p, f, margins: Optional[list] = None) -> torch.Tensor:
    chosen, weights, margin = route(h, w, p, f["router"])
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in chosen.unique().tolist():
        rows, place = (chosen == e).nonzero(as_tuple=True)
        y = bounded_unit(h[rows], w, f"{p}e{e}.", f["expert"]["limit"]) if e < f["router"]["experts"] else h[rows]
        out[rows] += weights[rows, place, None] * y
    if f.get("shared"):
        out = out + bounded_unit(h, w, p + "shared.", f["shared"]["limit"])
    return out


def token_side(x, tokens, c, w, i) -> torch.Tensor:
    """What a layer's own slice of the tokens' side vectors adds to the stream, whose rows x it is gated by."""
    p, dim, eps = f"l{i}.side.", c["token_side"]["dim"], c["norm"]["eps"]
    e = w["side.embed"][torch.tensor(tokens)][:, i * dim:(i + 1) * dim]
    return rms_norm((gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T, w[p + "norm"], eps)


def forward(c: dict, w: Dict[str, torch.Tensor], tokens: List[int], after_runs: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab].  `after_runs` receives the stream after every layer, `margins` the routers' margins."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = c["norm"]["eps"]
    x = token_rows(c, w, tokens)
    kept: Dict[int, tuple] = {}
    for i, L in enumerate(c["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if L["type"] == "attention":
            y = windowed_attention(h, w, p + "mix.", m, kept, i)
        elif L["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps)
        else:
            y = two_mixers(h, w, p + "mix.", m, eps)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            x = x + rms_norm(experts(h, w, p + "mlp.", L["mlp"], margins), w[p + "norm2b"], eps)
        if c.get("token_side"):
            x = x + token_side(x, tokens, c, w, i)
        if after_runs is not None:
            after_runs.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
