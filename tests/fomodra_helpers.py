"""Small Fomodra configurations and random weights for the tests, made here (not by the library), and the comparison
rules (those of the Rarelorn tests)."""
from __future__ import annotations

import copy
import math
from typing import Dict, List

import torch

from rarelorn_helpers import check_rows, noise, tokens      # noqa: F401  (used by the tests through this module)


def moe(experts, top, ff, limit, identity=0, shared=None):
    r = dict(experts=experts, top=top)
    if identity:
        r["identity"] = identity
    m = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=r)
    if shared:
        m["shared"] = dict(ff=shared[0], limit=shared[1])
    return m


def rotation(rot):
    if not rot:
        return None
    r = dict(dims=rot[0], base=rot[1])
    if len(rot) > 2:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2]))
    return r


def heads(H, d, kv=None, vdim=None, rot=None, mask=None, scale=None, kv_from=None):
    m = dict(heads=H, dim=d, scale=scale if scale is not None else 1.7 / math.sqrt(d))
    for key, v in (("kv_heads", kv), ("vdim", vdim), ("rot", rotation(rot)), ("kv_from", kv_from)):
        if v is not None:
            m[key] = v
    if mask:
        m["mask"] = dict(size=mask)
    return m


def attn(*a, **k):
    return dict(type="attention", mixer=heads(*a, **k))


def latent(H, d, rot_dim, kv_rank, vdim=None, base=1e4, mask=None, scale=None):
    m = dict(heads=H, dim=d, rot_dim=rot_dim, kv_rank=kv_rank, scale=scale if scale is not None else 1.7 / math.sqrt(d + rot_dim))
    if vdim is not None:
        m["vdim"] = vdim
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
    if mask:
        m["mask"] = dict(size=mask)
    return dict(type="latent_attention", mixer=m)


def parallel(left, inner, state, rank, conv):
    return dict(type="parallel", mixer=dict(left=left, right=dict(inner=inner, state=state, dt_rank=rank, conv=conv)))


def layer(mixer, mlp):
    return dict(mlp=mlp, **mixer)


def config(vocab, width, eps, layers, pairs=None, side=None):
    c = dict(architecture="Fomodra", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if pairs:
        c["embedding"] = dict(bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), pairs)))
    if side:
        c["token_side"] = dict(dim=side)
    return c


# K1: windows and chunks shorter than a page, a borrower whose window is wider than its lender's, values wider than keys, a layer
#     without a feed-forward, side vectors of 10.
# K2: sizes that are no multiple of 8 (general kernels), no rotation, no masks, no identity experts, one expert of five, one tap,
#     neither rows of token pairs nor side vectors.
# K3: every tensor-core kernel (heads of 64 / 64, 64 / 128, 64 + 16 / 80), masks over page borders, scaled rotation, two borrowers of
#     one layer, one of them without a window.
# K4: heads of 128 / 64, 80 / 48, 128 / 128 and 40 / 24 (padded tiles), 130 states a channel, eight taps, every choice taken.
# K5: sixteen query heads to a key head, values of 160, 48 states a channel, a latent of 128 without a rotated part, five layers of
#     one kind after another, more identity experts than experts.
CONFIGS: Dict[str, dict] = {
    "K1": config(150, 64, 1e-6,
                 [layer(attn(6, 16, kv=2, rot=(8, 5e4), mask=24), moe(6, 2, 24, 1.0, identity=2, shared=(40, 1.5))),
                  layer(parallel(heads(4, 16, kv=2, vdim=32, rot=(16, 1e4, (4.0, 1.0, 4.0, 64)), mask=20), 40, 6, 5, 3), None),
                  layer(attn(3, 16, kv=1, vdim=32, rot=(4, 1e3), mask=9), moe(4, 1, 32, 0.7, identity=1, shared=(24, 0.6))),
                  layer(latent(3, 16, 8, 24, vdim=8, mask=17), moe(5, 3, 16, 1.2, identity=3)),
                  layer(attn(2, 16, kv=2, rot=(8, 5e4), mask=70, kv_from=0), moe(4, 2, 40, 2.0, shared=(16, 1.0)))],
                 pairs=(53, 13, 7), side=10),
    "K2": config(131, 54, 1e-5,
                 [layer(attn(3, 10, vdim=14), moe(6, 3, 20, 1.0, shared=(36, 1.4))),
                  layer(parallel(heads(2, 14, kv=1, vdim=10), 30, 5, 3, 1), moe(5, 1, 36, 0.8)),
                  layer(latent(5, 6, 10, 18, vdim=14), None)]),
    "K3": config(300, 128, 2e-6,
                 [layer(attn(6, 64, kv=1, rot=(64, 1e5), mask=100), moe(16, 4, 32, 1.0, identity=3, shared=(64, 1.5))),
                  layer(parallel(heads(2, 64, vdim=128, rot=(32, 5e4, (8.0, 1.0, 4.0, 96)), mask=70), 160, 24, 12, 4), moe(8, 2, 64, 1.3, identity=1)),
                  layer(latent(4, 64, 16, 64, vdim=80, base=1e6, mask=65), moe(4, 2, 48, 1.0, shared=(96, 0.9))),
                  layer(attn(4, 64, kv=1, rot=(64, 1e5), mask=30, kv_from=0), moe(8, 3, 32, 1.1, identity=2, shared=(32, 1.2))),
                  layer(attn(2, 64, kv=1, rot=(64, 1e5), kv_from=0), None)],
                 pairs=(97, 31, 11), side=24),
    "K4": config(97, 80, 1e-5,
                 [layer(parallel(heads(3, 80, kv=1, vdim=48, rot=(40, 3e4), mask=64), 48, 130, 40, 8), moe(3, 5, 24, 1.0, identity=2, shared=(40, 1.0))),
                  layer(attn(4, 128, kv=2, vdim=64, rot=(128, 1e4), mask=65), moe(3, 3, 40, 1.6)),
                  layer(parallel(heads(2, 40, kv=2, vdim=24, rot=(8, 1e3), mask=33), 88, 16, 9, 2), None),
                  layer(latent(2, 128, 64, 128, vdim=128, mask=150), moe(4, 3, 16, 1.0, identity=1))],
                 pairs=(211, 5, 3), side=7),
    "K5": config(180, 96, 3e-6,
                 [layer(attn(16, 16, kv=1, rot=(2, 1e4), mask=40), moe(2, 3, 16, 1.0, identity=5, shared=(28, 1.1))),
                  layer(parallel(heads(3, 12, vdim=160, rot=(6, 1e3), mask=90), 72, 48, 17, 5), moe(9, 2, 28, 1.0)),
                  layer(latent(5, 24, 0, 128, vdim=32, mask=128), moe(6, 2, 32, 0.5, identity=2, shared=(24, 2.0))),
                  layer(attn(2, 32, kv=1, rot=(32, 500.0), mask=9), None),
                  layer(attn(4, 32, kv=1, rot=(32, 500.0), mask=150, kv_from=3), moe(4, 1, 24, 1.0, identity=1))],
                 pairs=(17, 3, 0), side=16),
}


def every_expert(c: dict) -> dict:
    """The configuration with every choice of every layer taken: no router's choice can turn on a rounding."""
    c = copy.deepcopy(c)
    for L in c["layers"]:
        if L["mlp"]:
            r = L["mlp"]["router"]
            r["top"] = r["experts"] + r.get("identity", 0)
    return c


def tensor_shapes(c: dict) -> Dict[str, List[int]]:
    W, n = c["width"], len(c["layers"])
    out = {"embed": [c["vocab"], W], "final.norm": [W], "head": [c["vocab"], W]}
    if c.get("embedding"):
        out["bigram"] = [c["embedding"]["bigram"]["buckets"] + 1, W]
    side = (c.get("token_side") or {}).get("dim")
    if side:
        out["side.embed"] = [c["vocab"], n * side]

    def attention(x, m, biases):
        H, d = m["heads"], m["dim"]
        G, dv = m.get("kv_heads", H), m.get("vdim", d)
        out.update({x + "q": [H * d, W], x + "o": [W, H * dv]})
        rows = [("q", H * d)]
        if m.get("kv_from") is None:
            out.update({x + "k": [G * d, W], x + "v": [G * dv, W]})
            rows += [("k", G * d), ("v", G * dv)]
        if biases:
            out.update({x + "sink": [H], **{x + k + ".b": [r] for k, r in rows}})

    for i, L in enumerate(c["layers"]):
        m, p = L["mixer"], f"l{i}."
        x = p + "mix."
        out.update({p + "norm1": [W], p + "norm1b": [W]})
        if L["type"] == "attention":
            attention(x, m, True)
        elif L["type"] == "latent_attention":
            H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m.get("vdim", m["dim"]), m["kv_rank"]
            out.update({x + "q": [H * (d + r), W], x + "dkv": [R + r, W], x + "dkv.norm": [R], x + "uk": [H * d, R], x + "uv": [H * dv, R],
                        x + "sink": [H], x + "g": [H, W], x + "o": [W, H * dv]})
        else:
            attention(x + "left.", m["left"], False)
            I, N, R, J = (m["right"][k] for k in ("inner", "state", "dt_rank", "conv"))
            y = x + "right."
            out.update({y + "in": [2 * I, W], y + "conv": [I, J], y + "conv.b": [I], y + "x": [R + 2 * N, I], y + "dt": [I, R], y + "dt.b": [I],
                        y + "A_log": [I, N], y + "D": [I], y + "o": [W, I], x + "left.out": [W], x + "right.out": [W]})
        if side:
            out.update({p + "side.gate": [side, W], p + "side.proj": [W, side], p + "side.norm": [W]})
        f = L["mlp"]
        if f is None:
            continue
        y, total = p + "mlp.", f["router"]["experts"] + f["router"].get("identity", 0)
        out.update({p + "norm2": [W], p + "norm2b": [W], y + "router": [total, W], y + "correction": [total]})
        units = [(f"{y}e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        if f.get("shared"):
            units.append((y + "shared.", f["shared"]["ff"]))
        for u, ff in units:
            out.update({u + "gate": [ff, W], u + "up": [ff, W], u + "down": [W, ff]})
    return out


def random_weights(c: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bfloat16-representable float32 tensors: matrices ~ N(0, 1.3^2 / fan_in), routers that spread their logits, corrections that
    turn choices, step sizes and decays between forgetting at once and keeping for hundreds of tokens, everything the design
    could leave at 1 or nought set to something else."""
    g = torch.Generator().manual_seed(seed)
    r = lambda s: torch.randn(*s, generator=g)
    out = {}
    for name, shape in tensor_shapes(c).items():
        end = name.split(".")[-1]
        if end in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out", "D"):
            t = 1.0 + 0.25 * r(shape)
        elif end == "conv":
            t = 0.4 * r(shape)
            t[:, -1] += 1.0
        elif name.endswith("dt.b"):
            t = -2.5 + 1.5 * r(shape)
        elif end == "A_log":
            t = 0.8 * r(shape)
        elif end == "sink":
            t = 0.5 + r(shape)
        elif end == "correction":
            t = 0.2 * r(shape)
        elif end == "b":
            t = 0.4 * r(shape)
        elif end == "router":
            t = r(shape) * 2.5 / math.sqrt(shape[1])
        elif name in ("bigram", "side.embed"):
            t = 0.8 * r(shape)
        else:
            t = r(shape) * 1.3 / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16).float()
    return out
