"""Small Rarelorn configurations and random weights for the tests, made here (not by the library), and the
comparison rules."""
from __future__ import annotations

import copy
import math
from typing import Dict, List, Optional

import torch

from tazizen_helpers import row_errors


def moe(experts, top, ff, groups=None, scale=None):
    r = dict(experts=experts, top=top)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    if scale is not None:
        r["scale"] = scale
    return dict(kind="moe", expert=dict(ff=ff), router=r)


def delta(heads, dim, vdim=None, kv=None, conv=4):
    m = dict(heads=heads, dim=dim)
    if vdim is not None:
        m["vdim"] = vdim
    if kv is not None:
        m["kv_heads"] = kv
    if conv:
        m["conv"] = conv
    return dict(type="delta", mixer=m)


def mlstm(heads, dim, vdim=None, cap=15.0):
    m = dict(heads=heads, dim=dim, gate_cap=cap)
    if vdim is not None:
        m["vdim"] = vdim
    return dict(type="mlstm", mixer=m)


def parallel(heads, dim, r_heads, r_dim, kv=None, vdim=None, rot=None, window=None, conv=4, scale=None, cap=12.0, left=0.9, right=1.1):
    l = dict(heads=heads, dim=dim, scale=scale if scale is not None else 1.7 / math.sqrt(dim))
    if kv is not None:
        l["kv_heads"] = kv
    if vdim is not None:
        l["vdim"] = vdim
    if rot:
        l["rot"] = dict(dims=rot[0], base=rot[1])
    if window:
        l["mask"] = dict(size=window)
    if conv:
        l["conv"] = conv
    if cap:
        l["softcap"] = cap
    return dict(type="parallel", mixer=dict(left=l, right=dict(heads=r_heads, dim=r_dim), left_scale=left, right_scale=right))


def layer(mixer, mlp):
    return dict(mlp=mlp, **mixer)


def config(vocab, width, eps, layers, loop=None):
    c = dict(architecture="Rarelorn", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


# Q1: a loop in the middle run three times, windows shorter than a page, values wider than keys, two value heads to a key head,
#     a layer without a feed-forward, convolutions of 4 and 3 taps.
# Q2: sizes that are no multiple of 8 (general kernels), no loop, no window, no rotation, no bound on the scores, one expert
#     of five, a convolution of two taps and none.
# Q3: every tensor-core kernel (heads of 64 / 64 and 128 / 128), a loop at the start, windows over page borders, two of four groups.
# Q4: heads of 80 / 48 and 48 / 160 (padded tiles), a loop at the end run once, five taps, one group, every expert chosen.
# Q5: recurrent heads of 16, 72, 130 and 8 channels (every size class of the scan and what lies between), sixteen query heads to a
#     key head, a rotation of one pair, eight taps, one tap.
CONFIGS: Dict[str, dict] = {
    "Q1": config(150, 64, 1e-6,
                 [layer(delta(4, 16, vdim=24, kv=2), moe(8, 2, 24, groups=(4, 2), scale=2.5)),
                  layer(parallel(4, 16, 3, 20, kv=2, vdim=32, rot=(8, 5e4), window=24, conv=3, left=0.6, right=1.3), None),
                  layer(mlstm(2, 24, vdim=40), moe(6, 2, 40, groups=(3, 1), scale=0.7)),
                  layer(parallel(2, 32, 2, 32, kv=1, rot=(32, 500.0), window=9), moe(4, 1, 32))],
                 loop=(1, 3, 3)),
    "Q2": config(131, 54, 1e-5,
                 [layer(parallel(3, 10, 5, 6, vdim=14, conv=2, cap=None, left=1.0, right=0.5), moe(6, 3, 20, groups=(3, 2))),
                  layer(mlstm(3, 18, vdim=10, cap=4.0), moe(5, 1, 36)),
                  layer(delta(3, 22, vdim=14, conv=None), None)]),
    "Q3": config(300, 128, 2e-6,
                 [layer(parallel(4, 64, 2, 64, kv=2, rot=(32, 1e5), window=100), moe(16, 4, 32, groups=(4, 2), scale=1.5)),
                  layer(delta(2, 64, vdim=64), moe(8, 2, 64)),
                  layer(parallel(2, 128, 1, 128, kv=2, rot=(64, 1e4), window=65, left=1.4, right=0.7), moe(4, 2, 48, groups=(2, 1), scale=3.0)),
                  layer(mlstm(1, 128, vdim=128), None)],
                 loop=(0, 2, 2)),
    "Q4": config(97, 80, 1e-5,
                 [layer(parallel(3, 80, 2, 40, kv=1, vdim=48, rot=(40, 3e4), window=64, conv=5), moe(4, 4, 24, groups=(1, 1), scale=2.0)),
                  layer(delta(6, 48, vdim=32, kv=2, conv=5), moe(3, 2, 40)),
                  layer(parallel(2, 48, 4, 24, vdim=160, rot=(48, 1e4), window=150, cap=30.0), None)],
                 loop=(1, 3, 1)),
    "Q5": config(180, 96, 3e-6,
                 [layer(parallel(16, 16, 6, 72, kv=1, rot=(2, 1e4), window=40, conv=8), moe(12, 5, 16, groups=(3, 2))),
                  layer(delta(2, 130, vdim=20, conv=8), moe(9, 2, 28, groups=(3, 1))),
                  layer(mlstm(5, 8, vdim=72), None),
                  layer(delta(3, 16, vdim=96, kv=1, conv=1), moe(8, 3, 32, groups=(2, 2), scale=0.5))],
                 loop=(0, 4, 2)),
}


def every_expert(c: dict) -> dict:
    """The configuration with every expert of every layer chosen: no router's choice can turn on a rounding."""
    c = copy.deepcopy(c)
    for L in c["layers"]:
        if L["mlp"]:
            r = L["mlp"]["router"]
            r["top"] = r["experts"]
            r.pop("groups", None)
    return c


def tensor_shapes(c: dict, rank: int = 6) -> Dict[str, List[int]]:
    W = c["width"]
    out = {"embed": [c["vocab"], W], "final.norm": [], "head": [c["vocab"], W]}
    loop = c.get("loop")
    if loop and loop["start"] < loop["stop"]:
        out["loop.step"] = [loop["times"], W]
    for i, L in enumerate(c["layers"]):
        m, p = L["mixer"], f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = []
        if L["type"] == "delta":
            H, d = m["heads"], m["dim"]
            G, dv = m.get("kv_heads", H), m.get("vdim", d)
            out.update({x + "q": [G * d, W], x + "k": [G * d, W], x + "v": [H * dv, W], x + "g": [H * dv, W], x + "b": [H, W], x + "a": [H, W],
                        x + "dt_bias": [H], x + "A_log": [H], x + "norm": [dv], x + "o": [W, H * dv]})
            if m.get("conv"):
                out.update({x + "q.conv": [G * d, m["conv"]], x + "k.conv": [G * d, m["conv"]], x + "v.conv": [H * dv, m["conv"]]})
        elif L["type"] == "mlstm":
            H, d = m["heads"], m["dim"]
            dv = m.get("vdim", d)
            out.update({x + "q": [H * d, W], x + "k": [H * d, W], x + "v": [H * dv, W], x + "g": [H * dv, W], x + "i": [H, W], x + "i.b": [H],
                        x + "f": [H, W], x + "f.b": [H], x + "norm": [H * dv], x + "o": [W, H * dv]})
        else:
            l, r = m["left"], m["right"]
            H, d = l["heads"], l["dim"]
            G, dv = l.get("kv_heads", H), l.get("vdim", d)
            y = x + "left."
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out.update({y + n: [rows, W], y + n + ".b": [rows]})
                if l.get("conv"):
                    out[y + n + ".conv"] = [rows, l["conv"]]
            out.update({y + "o": [W, H * dv], y + "o.b": [W], y + "temp": [H], y + "pb": [H]})
            z, D = x + "right.", r["heads"] * r["dim"]
            out.update({z + "mu." + n: [W] for n in "rkvgw"})
            out.update({z + n: [D, W] for n in "rkvg"})
            out.update({z + "w1": [rank, W], z + "w2": [D, rank], z + "w0": [D], z + "u": [r["heads"], r["dim"]], z + "norm": [D], z + "o": [W, D]})
        f = L["mlp"]
        if f is None:
            continue
        out[p + "norm2"] = []
        y, ff = p + "mlp.", f["expert"]["ff"]
        for e in range(f["router"]["experts"]):
            out.update({f"{y}e{e}.gate": [ff, W], f"{y}e{e}.up": [ff, W], f"{y}e{e}.down": [W, ff]})
        out[y + "router"] = [f["router"]["experts"], W]
    return out


def random_weights(c: dict, seed: int = 0, rank: int = 6) -> Dict[str, torch.Tensor]:
    """bfloat16-representable float32 tensors: matrices ~ N(0, 1.3^2 / fan_in), routers that spread their logits, decays between
    forgetting at once and keeping for hundreds of tokens, convolutions that lean on the current token, everything the design
    could leave at 1 or nought set to something else."""
    g = torch.Generator().manual_seed(seed)
    r = lambda s: torch.randn(*s, generator=g) if s else torch.randn((), generator=g)
    out = {}
    for name, shape in tensor_shapes(c, rank).items():
        end = name.split(".")[-1]
        if end in ("norm1", "norm2") or name == "final.norm" or end in ("norm", "temp"):
            t = 1.0 + 0.2 * r(shape)
        elif end == "conv":
            t = 0.4 * r(shape)
            t[:, -1] += 1.0
        elif ".mu." in name:
            t = torch.rand(shape, generator=g)
        elif end == "w0":
            t = -2.0 + 1.5 * r(shape)
        elif end == "dt_bias":
            t = -3.0 + 1.5 * r(shape)
        elif end == "A_log":
            t = 0.5 * r(shape)
        elif name.endswith("f.b"):
            t = 3.0 + 1.5 * r(shape)
        elif name.endswith("i.b") or end == "u" or name == "loop.step":
            t = 0.7 * r(shape)
        elif end == "pb":
            t = -1.5 + 0.7 * r(shape)
        elif end == "b" and len(shape) == 1:
            t = 0.3 * r(shape)
        elif end == "router":
            t = r(shape) * 3.0 / math.sqrt(shape[1])
        else:
            t = r(shape) * 1.3 / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16).float()
    return out


def tokens(c: dict, n: int, seed: int) -> List[int]:
    g = torch.Generator().manual_seed(9000 + seed)
    return torch.randint(0, c["vocab"], (n,), generator=g).tolist()


# float32: rounding alone, except behind a router's choice that is closer than that (such positions and those that see them
# test nothing).  bfloat16 runs of whole models have every expert chosen (every_expert), so that rounding alone is left; the
# choice itself is compared mechanism by mechanism.  How much a rounding weighs differs from position to position: where a
# recurrent read-out is all but cancelled (above all at a first token whose key and query are nearly orthogonal) the norm behind
# it divides by almost nothing and even the sign hangs on the last bits, and the tokens after it see that.  So bfloat16 is
# compared with room for what the plain implementation itself does under roundings of the same size (`noise`).
TOL = {"float32": 1e-4, "bfloat16": 0.12}
NOISE_ROOM = 3.0


def noise(plain_forward, c: dict, w: Dict[str, torch.Tensor], toks: List[int], ref: torch.Tensor, runs: int = 8) -> torch.Tensor:
    """Per position: the largest row error of plain runs whose matrices are off by about a bfloat16 rounding at random."""
    worst = torch.zeros(len(toks), dtype=torch.float64)
    for k in range(runs):
        g = torch.Generator().manual_seed(k)
        off = {n: v * (1 + torch.randn(v.shape, generator=g) * 2.0 ** -8) if v.dim() > 1 else v for n, v in w.items()}
        worst = torch.maximum(worst, row_errors(plain_forward(c, off, toks), ref))
    return worst


def check_rows(got: torch.Tensor, ref: torch.Tensor, dtype: str, what: str, margin: Optional[torch.Tensor] = None,
               rounding: Optional[torch.Tensor] = None) -> None:
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: logits are not finite"
    e = row_errors(got, ref)
    limit = torch.full_like(e, TOL[dtype])
    if dtype == "bfloat16":
        if rounding is not None:
            limit = limit + NOISE_ROOM * rounding
    elif margin is not None:
        unsure = (margin <= 2e-4).nonzero()
        if unsure.numel():
            e, limit = e[:int(unsure[0])], limit[:int(unsure[0])]
    if e.numel() == 0:
        return
    worst = int((e / limit).argmax())
    assert float(e[worst]) < float(limit[worst]), f"{what}: row error {float(e[worst]):.3e}, limit {float(limit[worst]):.3e} at position {worst} of {e.numel()} ({dtype})"
