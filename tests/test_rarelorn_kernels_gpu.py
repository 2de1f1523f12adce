"""The mechanisms Rarelorn adds, each alone against the plain implementation's function for it: attention whose weights stand
for themselves in all three kernels (with single keys that stand out at page borders and on either side of a window's edge, and
with every key counting), the convolution, rotation and placement in one pass, the three recurrences with their convolutions,
token shift, gates and carried state, mixers side by side, a norm with one gain, the additions at a pass's start, softmax
routing among groups.  Prompts, portions and single tokens share the calls."""
import math

import pytest
import torch

import plain_rarelorn as P
import rarelorn_helpers as S
from test_parts_gpu import PAGE, Step, act, part
from test_sobezen_kernels_gpu import LENS, N_PAGES, PAGE_OF, PORTIONS, bf, close

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
EPS, WIDTH = 1e-5, 56


def ops():
    from libllm_b200.csrc import ops as o
    return o


# ---------------------------------------------------------------- attention whose weights stand for themselves
def paged(kd, vd, tdt, seed=0):
    """keys [T, G, d], values [T, G, dv] -> stores and the page table, pages scattered"""
    T, G, d = kd.shape
    n = (T + PAGE - 1) // PAGE
    pages = torch.randperm(n + 3, generator=torch.Generator().manual_seed(seed))[:n]
    kc = torch.full((n + 3, G, PAGE, d), 7.0).to(tdt).to(DEV)           # other pages: finite numbers that would show
    vc = torch.full((n + 3, G, PAGE, vd.shape[2]), 50.0).to(tdt).to(DEV)
    for t in range(T):
        kc[pages[t // PAGE], :, t % PAGE] = kd[t].to(tdt).to(DEV)
        vc[pages[t // PAGE], :, t % PAGE] = vd[t].to(tdt).to(DEV)
    return kc, vc, pages.to(torch.int32)[None].to(DEV)


def run_attention(form, q, kc, vc, table, rows, H, G, window, scale, temp, bias, cap, out_scale, n_splits=1):
    """the queries at positions `rows` (contiguous) of one sequence"""
    i32 = dict(dtype=torch.int32, device=DEV)
    n = len(rows)
    out = torch.empty(n, H * vc.shape[3], dtype=q.dtype, device=DEV)
    o = ops()
    o.sigmoid_attention(form, q, out, kc, vc, torch.zeros(n, **i32), torch.tensor(rows, **i32), torch.tensor([0, n], **i32),
                        torch.tensor([rows[0]], **i32), table, n, H, G, window, scale, temp.to(DEV), bias.to(DEV), cap, out_scale, n_splits)
    o.check_tc_status()
    return out.float().cpu()


SIZES = [(4, 2, 64, 64), (2, 2, 128, 128), (3, 1, 80, 48), (4, 2, 48, 160), (16, 1, 16, 16), (2, 1, 96, 240), (8, 2, 112, 64), (6, 3, 32, 112)]


@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("window", [None, 50, 64, 65, 130])
def test_one_key_that_stands_out(sizes, window):
    """All weights but one are nought (a bias far below); the one key that matches its query lies somewhere else for
    every query: at the window's last visible position, just outside it, at a page's first and last position, at the query's own
    place, far back.  The result is that key's value, or nought."""
    H, G, d, dv = sizes
    T, scale = 210, 1.0
    g = torch.Generator().manual_seed(d + dv)
    codes = torch.sign(torch.randn(T, d, generator=g))                  # q . k = d where they match, about sqrt(d) elsewhere
    k = codes[:, None, :].expand(T, G, d).clone()
    v = bf(torch.randn(T, G, dv, generator=g))
    W = window or 10 ** 6
    target = []
    for i in range(T):
        options = [i, i - W + 1, i - W, i // PAGE * PAGE, i // PAGE * PAGE - 1, i - 37, 0]
        target.append(min(max(options[i % 7], 0), i))
    q = codes[torch.tensor(target)][:, None, :].expand(T, H, d).reshape(T, H * d)
    bias = torch.full((H,), -0.75 * d)
    temp = torch.ones(H)
    # codes that happen to lie close: counted with their own weights
    s = (codes[torch.tensor(target)].double() @ codes.double().T)
    wts = torch.sigmoid(s - 0.75 * d) * P.visible(T, window)
    ref = torch.einsum("ij,jgc->igc", wts, v.double()).repeat_interleave(H // G, dim=1).reshape(T, H * dv) * 1.5
    for dtype in DTYPES:
        tdt = DT[dtype]
        kc, vc, table = paged(k, v, tdt, seed=3)
        qd = q.to(tdt).to(DEV)
        forms = ["generic"] + (["prompt"] if dtype == "bfloat16" else [])
        for form in forms:
            for a, b in ((0, T), (64, T), (63, 130), (129, 131), (T - 1, T)):
                got = run_attention(form, qd[a:b].contiguous(), kc, vc, table, list(range(a, b)), H, G, window, scale, temp, bias, 0.0, 1.5)
                assert float((got - ref[a:b]).abs().max()) < 0.04, f"{form} {dtype} rows {a}..{b}"
        if dtype == "bfloat16":
            for i in list(range(60, 70)) + list(range(126, 134)) + [0, 1, T - 1]:
                for n_splits in (1, 2, 4):
                    got = run_attention("single", qd[i:i + 1].contiguous(), kc, vc, table, [i], H, G, window, scale, temp, bias, 0.0, 1.5, n_splits)
                    assert float((got - ref[i:i + 1]).abs().max()) < 0.04, f"single token at {i}, {n_splits} runs"


@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("cap", [0.0, 5.0, 30.0])
def test_every_key_counts(sizes, cap):
    """Random scores, temperatures and biases per head, with and without the bound, against the plain weights."""
    H, G, d, dv = sizes
    T, window, scale, out_scale = 333, 100, 1.6 / math.sqrt(d), 0.7
    g = torch.Generator().manual_seed(d * 3 + dv)
    q, k, v = bf(2 * torch.randn(T, H, d, generator=g)), bf(torch.randn(T, G, d, generator=g)), bf(torch.randn(T, G, dv, generator=g))
    temp, bias = 1 + 0.4 * torch.randn(H, generator=g), torch.randn(H, generator=g)
    see = P.visible(T, window)
    heads = []
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        heads.append(P.sigmoid_weights(s, see, temp[h].double(), cap, bias[h].double()) @ v[:, h // (H // G)].double())
    ref = torch.cat(heads, 1) * out_scale
    spread = ref.abs().mean()
    for dtype in DTYPES:
        tdt = DT[dtype]
        kc, vc, table = paged(k, v, tdt)
        qd = q.reshape(T, H * d).to(tdt).to(DEV)
        for form in ["generic"] + (["prompt"] if dtype == "bfloat16" else []):
            got = run_attention(form, qd, kc, vc, table, list(range(T)), H, G, window, scale, temp, bias, cap, out_scale)
            err = float((got - ref).abs().max() / spread)
            assert err < (2e-5 if dtype == "float32" else 0.06), f"{form} {dtype}: {err:.2e}"
            one = run_attention(form, qd[T - 3:T - 2].contiguous(), kc, vc, table, [T - 3], H, G, window, scale, temp, bias, cap, out_scale)
            assert float((one - got[T - 3]).abs().max() / spread) < (1e-6 if dtype == "float32" else 0.02)
        if dtype == "bfloat16":
            for i in (0, 5, 99, 100, 200, 332):
                for n_splits in (1, 3):
                    got = run_attention("single", qd[i:i + 1].contiguous(), kc, vc, table, [i], H, G, window, scale, temp, bias, cap, out_scale, n_splits)
                    assert float((got - ref[i:i + 1]).abs().max() / spread) < 0.06, f"single token at {i}, {n_splits} runs"


# ---------------------------------------------------------------- the mixers
def mixer_of(layers, i, dtype, seed, max_positions=1024):
    """Layer i's mixer of a model of `layers`, as the configuration's reader describes it, with weights of its own."""
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, layers)
    spec = _lib.describe_model(c, dtype)["spec"]["layers"][i]["mixer"]
    w = {k: v for k, v in S.random_weights(c, seed).items() if k.startswith(f"l{i}.mix.")}
    return spec, w


def built(spec, w, dtype, max_positions=1024):
    m = part("mixer", spec, dtype, max_positions)
    m.load(w)
    return m


class Runner:
    """A mixer with a cache and state of its own, run over sequences that bring portions; sequence b lives in slot slots[b]."""

    def __init__(self, m, dtype, n_slots=5):
        self.m, self.dtype = m, dtype
        self.state, self.keep = [], []
        for s in m.description["state"]:
            t = torch.zeros(n_slots, *s["shape"], dtype=DT[s["dtype"]], device=DEV)
            self.keep.append(t)
            self.state.append(dict(name=s["name"], ptr=t.data_ptr(), shape=s["shape"], dtype=s["dtype"], n_slots=n_slots))
        c = m.description["cache"]
        self.store = None
        if c:
            make = lambda d: torch.zeros(N_PAGES, c["n_kv_heads"], PAGE, d, dtype=DT[dtype], device=DEV)
            self.store = (make(c["k_dim"]), make(c["v_dim"]))

    def run(self, x, portions, lens, slots=(3, 0, 2, 4)):
        done, got = [0] * len(lens), [[] for _ in lens]
        for por in portions:
            seqs = [b for b in range(len(lens)) if por[b] > 0]
            step = Step([por[b] for b in seqs], [done[b] for b in seqs])
            step.keep["seq_slot"].copy_(torch.tensor([slots[b] for b in seqs], dtype=torch.int32))
            step.json["slots"] = [slots[b] for b in seqs]
            width = max((done[b] + por[b] + PAGE - 1) // PAGE for b in seqs)
            table = torch.tensor([[PAGE_OF[(b, j)] for j in range(width)] for b in seqs], dtype=torch.int32, device=DEV)
            xs = torch.cat([x[b][done[b]:done[b] + por[b]] for b in seqs]).to(DT[self.dtype]).to(DEV)
            call = dict(step=step.json, x=act(xs), state=self.state)
            if self.store:
                call["cache"] = dict(k=self.store[0].data_ptr(), v=self.store[1].data_ptr(), n_pages=N_PAGES, page_table=table.data_ptr(),
                                     table_width=width, writes=True)
            res = self.m.forward(call)
            out = res["out"].torch().float()
            out = out.sum(0) if out.dim() == 3 else out
            if res.get("out_bias") is not None:
                out = out + res["out_bias"].torch()
            out, at = out.cpu(), 0
            for b in seqs:
                got[b].append(out[at:at + por[b]])
                at += por[b]
                done[b] += por[b]
        assert done == list(lens)
        return [torch.cat(r) for r in got]


def inputs(seed, lens=LENS):
    g = torch.Generator().manual_seed(seed)
    return [bf(torch.randn(n, WIDTH, generator=g)) for n in lens]


DELTA = [dict(heads=4, dim=16, vdim=24, kv=2, conv=4), dict(heads=3, dim=64, vdim=64, conv=3), dict(heads=2, dim=128, vdim=40, kv=1, conv=2),
         dict(heads=3, dim=22, vdim=13, conv=None), dict(heads=2, dim=130, vdim=20, conv=8), dict(heads=6, dim=8, vdim=136, kv=1, conv=1),
         dict(heads=2, dim=256, vdim=17, conv=5), dict(heads=1, dim=32, vdim=300, conv=4)]
MEMORY = [dict(heads=2, dim=24, vdim=40), dict(heads=3, dim=18, vdim=10, cap=4.0), dict(heads=2, dim=64, vdim=64), dict(heads=1, dim=128, vdim=128),
          dict(heads=5, dim=8, vdim=72), dict(heads=1, dim=200, vdim=31), dict(heads=3, dim=32, vdim=16, cap=30.0)]
MIXING = [dict(r_heads=3, r_dim=20), dict(r_heads=2, r_dim=64), dict(r_heads=1, r_dim=128), dict(r_heads=6, r_dim=6), dict(r_heads=2, r_dim=72),
          dict(r_heads=1, r_dim=256)]
LEFT = [dict(heads=4, dim=16, kv=2, vdim=32, rot=(8, 5e4), window=24, conv=3), dict(heads=3, dim=10, vdim=14, conv=2, cap=None),
        dict(heads=4, dim=64, kv=2, rot=(32, 1e5), window=100), dict(heads=2, dim=128, kv=2, rot=(128, 1e4), window=65),
        dict(heads=3, dim=80, kv=1, vdim=48, rot=(40, 3e4), window=64, conv=5), dict(heads=2, dim=48, vdim=160, rot=(12, 1e4), conv=None),
        dict(heads=16, dim=16, kv=1, rot=(2, 1e4), window=130, conv=8), dict(heads=3, dim=12, vdim=300, rot=(6, 1e3), window=70, conv=4)]


def state_of_a_fresh_slot_is_used_again(r, x, ref, dtype, what, room):
    """The slots' state set to nought (as the cache manager does when a slot is taken), other sequences in them: the same results."""
    for t in r.keep:
        t.zero_()
    again = r.run([x[1], x[2], x[1]], [[66, 3, 1]] + [[0, 127, 64]] + [[0, 0, 1]], [66, 130, 66], slots=(0, 3, 4))
    close(again[0], ref[1], dtype, what + ", a slot used again", roundings=room)
    close(again[1], ref[2], dtype, what + ", a slot used again", roundings=room)
    close(again[2], ref[1], dtype, what + ", one token, then the rest", roundings=room)


# A read-out that is all but cancelled is divided by almost nothing: such rows are left out in bfloat16 (their share of the
# largest head differs from design to design, so the rows are found by what a rounding of the inputs does to the plain result).
def settled(fn, x, ref):
    g = torch.Generator().manual_seed(1)
    keep = torch.ones(len(ref), dtype=torch.bool)
    for _ in range(3):
        off = fn(x * (1 + torch.randn(x.shape, generator=g) * 2.0 ** -8))
        keep &= ((off - ref).abs() / (ref.abs() + ref.abs().mean())).max(-1).values < 0.06
    return keep


def check_mixer(spec, w, fn, seed, what, room32=4.0, room16=8.0):
    for dtype in DTYPES:
        r = Runner(built(spec, w, dtype), dtype)
        x = inputs(seed)
        ref = [fn(xb.double()) for xb in x]
        got = r.run(x, PORTIONS, LENS)
        for b in range(len(LENS)):
            keep = settled(fn, x[b].double(), ref[b]) if dtype == "bfloat16" else torch.ones(LENS[b], dtype=torch.bool)
            assert int(keep.sum()) > 0.5 * LENS[b], f"{what}: too few settled rows"
            close(got[b][keep], ref[b][keep], dtype, f"{what}, sequence {b}", roundings=room32 if dtype == "float32" else room16)
        if dtype == "float32":
            state_of_a_fresh_slot_is_used_again(r, x, ref, dtype, what, room32)
            # the same sequence cut other ways
            long_ = inputs(seed + 1, [200])
            whole = None
            for portions in ([[200]], [[1]] * 200, [[2]] * 100, [[150], [50]], [[7], [8], [9], [176]]):
                for t in r.keep:
                    t.zero_()
                out = r.run(long_, portions, [200], slots=(1,))[0]
                whole = out if whole is None else whole
                close(out, whole.double(), dtype, f"{what} cut as {portions[:2]}", roundings=room32)


@pytest.mark.parametrize("m", DELTA)
def test_gated_delta(m):
    layers = [S.layer(S.delta(**m), None)]
    spec, w = mixer_of(layers, 0, "float32", 5)
    wd = {k: v.double() for k, v in w.items()}
    check_mixer(spec, w, lambda h: P.delta(h, wd, "l0.mix.", layers[0]["mixer"], EPS), 11, f"gated delta {m}")


@pytest.mark.parametrize("m", MEMORY)
def test_matrix_memory(m):
    layers = [S.layer(S.mlstm(**m), None)]
    spec, w = mixer_of(layers, 0, "float32", 6)
    wd = {k: v.double() for k, v in w.items()}
    check_mixer(spec, w, lambda h: P.mlstm(h, wd, "l0.mix.", layers[0]["mixer"], EPS), 12, f"matrix memory {m}")


@pytest.mark.parametrize("m", MIXING)
def test_time_mixing(m):
    layers = [S.layer(S.parallel(1, 8, **m), None)]
    spec, w = mixer_of(layers, 0, "float32", 7)
    right = spec["mixers"][1]
    assert right["kind"] == "time_mixing" and right["out_scale"] == 1.1
    wr = {k: v for k, v in w.items() if ".right." in k}
    wd = {k: v.double() for k, v in wr.items()}
    check_mixer(right, wr, lambda h: 1.1 * P.time_mixing(h, wd, "l0.mix.right.", layers[0]["mixer"]["right"], EPS), 13, f"time mixing {m}")


@pytest.mark.parametrize("m", LEFT)
def test_sigmoid_attention_with_its_convolutions(m):
    layers = [S.layer(S.parallel(r_heads=1, r_dim=8, left=0.6, **m), None)]
    spec, w = mixer_of(layers, 0, "float32", 8)
    left = spec["mixers"][0]
    wl = {k: v for k, v in w.items() if ".left." in k}
    wd = {k: v.double() for k, v in wl.items()}
    check_mixer(left, wl, lambda h: 0.6 * P.attention(h, wd, "l0.mix.left.", layers[0]["mixer"]["left"]), 14, f"sigmoid attention {m}")


@pytest.mark.parametrize("m", [dict(LEFT[0], r_heads=3, r_dim=20), dict(LEFT[2], r_heads=2, r_dim=64, left=1.4, right=0.3), dict(LEFT[1], r_heads=2, r_dim=10)])
def test_two_mixers_side_by_side(m):
    layers = [S.layer(S.parallel(**m), None)]
    spec, w = mixer_of(layers, 0, "float32", 9)
    wd = {k: v.double() for k, v in w.items()}
    check_mixer(spec, w, lambda h: P.side_by_side(h, wd, "l0.mix.", layers[0]["mixer"], EPS), 15, f"side by side {m}")


def test_a_forgotten_past_stays_forgotten():
    """The memory's running maximum over large gates: an input gate at its bound after a long quiet stretch, and a forget gate at
    its lower bound, change the scale of everything before; the sums must follow without overflow."""
    layers = [S.layer(S.mlstm(2, 16, vdim=8, cap=40.0), None)]
    spec, w = mixer_of(layers, 0, "float32", 10)
    for n in ("i", "f"):
        w[f"l0.mix.{n}"] = bf(w[f"l0.mix.{n}"] * 20)              # log gates from one bound to the other
    wd = {k: v.double() for k, v in w.items()}
    r = Runner(built(spec, w, "float32"), "float32")
    x = inputs(16)
    got = r.run(x, PORTIONS, LENS)
    for b in range(len(LENS)):
        ref = P.mlstm(x[b].double(), wd, "l0.mix.", layers[0]["mixer"], EPS)
        close(got[b], ref, "float32", f"gates at their bounds, sequence {b}", roundings=30.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_state_belongs_to_its_slot(dtype):
    """Two sequences in turn, single tokens and portions, against each alone; a third slot's state is not touched."""
    layers = [S.layer(S.parallel(2, 16, 2, 16, window=20), None)]
    spec, w = mixer_of(layers, 0, dtype, 12)
    m = built(spec, w, dtype)
    x = inputs(17, [40, 40])
    both, alone = Runner(m, dtype), Runner(m, dtype)
    for t in both.keep:
        t[4] = 3.0
    got = both.run(x, [[10, 0], [0, 5], [1, 1], [1, 1], [28, 33]], [40, 40], slots=(1, 2))
    for t in both.keep:
        assert float((t[4].float() - 3.0).abs().max()) == 0 and float(t[0].float().abs().max()) == 0 and float(t[3].float().abs().max()) == 0
    for b in range(2):
        for t in alone.keep:
            t.zero_()
        one = alone.run([x[b]], [[40]], [40], slots=(0,))[0]
        close(got[b], one.double(), dtype, f"sequence {b} among others", roundings=1.0 if dtype == "float32" else 3.0)


# ---------------------------------------------------------------- norm with one gain, additions, routing
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_with_one_gain(dtype):
    norm = part("norm", dict(kind="rmsnorm", size=104, eps=3e-4, weight="n", one_gain=True), dtype)
    assert norm.description["tensor_needs"] == [dict(name="n", shape=[], role="vector", optional=False)]
    norm.load({"n": torch.tensor(1.375)})
    step = Step([5, 2], [0, 0])
    x = torch.randn(7, 104, device=DEV)
    out = norm.forward(dict(step=step.json, hidden=104, resid=x.clone().data_ptr(), pending=None))["out"].torch()
    close(out.float().cpu(), P.scalar_norm(x.cpu().double(), torch.tensor(1.375), 3e-4), dtype, "norm with one gain")


def test_what_a_pass_adds_to_its_input():
    """Models that differ only in the loop: what comes before a pass's first layer is the token rows (from the second pass on)
    and the pass's own vector."""
    from libllm_b200.engine import Engine
    from replay import replay_batch
    layers = [S.layer(S.delta(2, 16, conv=2), None), S.layer(S.mlstm(1, 16), None)]
    for loop in ((0, 1, 2), (1, 2, 3), (0, 2, 1), (0, 2, 2)):
        c = S.config(40, 32, EPS, layers, loop=loop)
        w = S.random_weights(c, 2)
        toks = S.tokens(c, 30, 1)
        got = replay_batch(Engine.from_tensors(c, w, dtype="float32", max_tokens=128), [("r", toks, 20)])["r"]
        S.check_rows(got, P.forward(c, w, toks), "float32", f"loop {loop}")


@pytest.mark.parametrize("E,top,groups,scale", [(16, 3, (2, 1), 1.5), (8, 4, (2, 1), 2.5), (6, 3, (3, 2), 1.0), (5, 1, None, 1.0), (12, 5, (3, 2), 0.5),
                                                 (4, 4, (1, 1), 2.0), (64, 6, (8, 3), 1.0), (9, 2, (9, 4), 1.0)])
def test_choice_by_softmax_scores_among_the_best_groups(E, top, groups, scale):
    g = torch.Generator().manual_seed(E * 10 + top)
    h = torch.randn(300, 32, generator=g).double()
    w = {"router": torch.randn(E, 32, generator=g).double() * 0.5}
    r = dict(experts=E, top=top, scale=scale)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    chosen, weights, margin = P.route(h, w, "", r)
    got_c, got_w = ops().moe_route_grouped((h @ w["router"].T).float().to(DEV), top, None, groups[0] if groups else 1, groups[1] if groups else 1, 1,
                                           score="softmax", renormalize=False, route_scale=scale)
    sure = margin > 1e-4
    assert int(sure.sum()) > 270
    assert torch.equal(got_c.cpu().long()[sure], chosen[sure])
    close(got_w.cpu()[sure], weights[sure], "float32", "weights")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("f", [S.moe(8, 4, 24, groups=(2, 1), scale=2.5), S.moe(6, 3, 20, groups=(3, 2)), S.moe(5, 1, 36), S.moe(16, 4, 32, groups=(4, 2), scale=0.5)])
def test_routed_feed_forward(f, dtype):
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, [S.layer(S.delta(2, 16), f)])
    spec = _lib.describe_model(c, dtype)["spec"]["layers"][0]["ff"]
    w = {k: v for k, v in S.random_weights(c, 8).items() if k.startswith("l0.mlp.")}
    ff = part("feed_forward", spec, dtype)
    ff.load(w)
    for T in (1, 7, 200):
        x = bf(torch.randn(T, WIDTH, generator=torch.Generator().manual_seed(T)))
        margins = []
        ref = P.experts(x.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", f, margins)
        out = ff.forward(dict(step=Step([T], [0]).json, x=act(x.to(DT[dtype]).to(DEV))))["out"].torch().float()
        out = (out.sum(0) if out.dim() == 3 else out).cpu()
        sure = margins[0] > (1e-4 if dtype == "float32" else 3e-2)
        if int(sure.sum()):
            close(out[sure], ref[sure], dtype, f"routed feed-forward, {T} tokens", roundings=4.0)
