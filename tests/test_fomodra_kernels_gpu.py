"""The mechanisms Fomodra adds, each alone against the plain implementation's function for it: results normed before they are
added (one, or two side by side), attention with biases, a sink per head, a window or chunks, values of another width, keys and
values borrowed from another run, latent attention with queries from the input, sinks and a gate per head, the selective scan with
its convolution and carried state, experts with a bounded unit among identity experts.  Attention is run with scores sharp enough
that one key stands out for most queries, and with a key planted just inside and just outside every mask; prompts, portions and
single tokens share the calls."""
import math

import pytest
import torch

import fomodra_helpers as S
import plain_fomodra as P
from test_parts_gpu import PAGE, Step, act, part, summed
from test_rarelorn_kernels_gpu import Runner, built, check_mixer
from test_sobezen_kernels_gpu import LENS, N_PAGES, PORTIONS, bf, close, run_in_portions

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
EPS, WIDTH = 1e-5, 56


# ---------------------------------------------------------------- results with norms of their own
@pytest.mark.parametrize("H", [48, 50, 1024, 2048, 2052, 4096, 4104, 6000])
@pytest.mark.parametrize("parts,first", [(1, 0), (3, 0), (9, 0), (17, 0), (2, 1), (7, 3), (16, 15)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_result_is_normed_before_it_is_added(H, parts, first, dtype):
    """The pass that adds: y (the sum of the parts, or half the sum of two normed results) over its root mean square, times a weight,
    into the stream; then the next norm.  All rows, and chosen rows, which leave the stream alone."""
    T = 5
    g = torch.Generator().manual_seed(H + parts)
    r = lambda *s: torch.randn(*s, generator=g)
    w = {"n": 1 + 0.2 * r(H)}
    x, y, post, wa, wb = r(T, H), r(parts, T, H) * 3, 1 + 0.2 * r(H), 1 + 0.2 * r(H), 1 + 0.2 * r(H)
    norm = part("norm", dict(kind="rmsnorm", size=H, eps=3e-4, weight="n"), dtype)
    norm.load(w)
    total = y.double().sum(0)
    if first:
        total = 0.5 * (P.rms_norm(y[:first].double().sum(0), wa.double(), 2e-3) + P.rms_norm(y[first:].double().sum(0), wb.double(), 2e-3))
    ref_x = x.double() + P.rms_norm(total, post.double(), 1e-2)
    ref = P.rms_norm(ref_x, w["n"].double(), 3e-4)
    dev = {k: v.contiguous().to(DEV) for k, v in dict(y=y, post=post, wa=wa, wb=wb).items()}
    pending = dict(ptr=dev["y"].data_ptr(), dtype="float32", rows=T, cols=H, parts=parts, part_stride=T * H, post=dev["post"].data_ptr(),
                   post_eps=1e-2)
    if first:
        pending.update(first_parts=first, pair_w=[dev["wa"].data_ptr(), dev["wb"].data_ptr()], pair_eps=2e-3, pair_scale=0.5)
    step = Step([T], [0])
    resid = x.to(DEV)
    rows = torch.tensor([4, 0, 2], dtype=torch.int32, device=DEV)
    out = norm.forward(dict(step=step.json, hidden=H, resid=resid.data_ptr(), pending=pending, rows=rows.data_ptr(), n_rows=3))
    close(out["out"].torch().float().cpu(), ref[[4, 0, 2]], dtype, "chosen rows", roundings=0.3)
    assert torch.equal(resid.cpu(), x)
    out = norm.forward(dict(step=step.json, hidden=H, resid=resid.data_ptr(), pending=pending))
    assert out["pending"] is None
    close(resid.cpu(), ref_x, "float32", "the stream", roundings=0.3)
    close(out["out"].torch().float().cpu(), ref, dtype, "the next norm", roundings=0.3)


# ---------------------------------------------------------------- attention
def mixers_of(layers, dtype, seed, sharpen=None):
    """The mixers of a model of `layers`, as the configuration's reader describes them, and their weights."""
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, layers)
    spec = _lib.describe_model(c, dtype)["spec"]["layers"]
    w = S.random_weights(c, seed)
    if sharpen:
        sharpen(w)
    mixers = []
    for i in range(len(layers)):
        m = part("mixer", spec[i]["mixer"], dtype, 1024)
        m.load({k: v for k, v in w.items() if k.startswith(f"l{i}.mix.")})
        mixers.append(m)
    return mixers, {k: v.double() for k, v in w.items()}, spec


def stores(m, dtype):
    c = m.description["cache"]
    make = lambda d: torch.zeros(N_PAGES, c["n_kv_heads"], PAGE, d, dtype=DT[dtype], device=DEV) if d else None
    return make(c["k_dim"]), make(c["v_dim"])


def inputs(seed, lens=LENS):
    g = torch.Generator().manual_seed(seed)
    return [bf(torch.randn(n, WIDTH, generator=g)) for n in lens]


# heads, key heads, head size, value size, rotation, window: exact tiles, padded ones, sizes of the general kernel alone, groups from
# one to sixteen, windows shorter than a page, of a page, over several, none
SIZES = [(6, 1, 64, 64, (64, 1e4), 100), (4, 2, 128, 128, (64, 1e4), 65), (8, 2, 32, 32, (16, 1e3), 64), (3, 1, 80, 48, (40, 3e3), 150),
         (2, 2, 64, 128, (32, 1e4, (4.0, 1.0, 4.0, 64)), 70), (16, 1, 16, 16, (2, 1e4), 9), (4, 1, 40, 24, (8, 1e3), None),
         (2, 1, 128, 64, (128, 1e4), 33), (3, 3, 10, 14, None, 20), (2, 1, 24, 160, (12, 500.0), 128), (5, 1, 24, 24, (24, 1e4), 90), (2, 1, 64, 64, None, 50)]


@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_windowed_attention_with_sinks_and_a_borrower(sizes, dtype):
    """Three sequences at once through a run with keys of its own and one that borrows them, with another window (wider, narrower or
    none) and queries of its own."""
    H, G, d, dv, rot, window = sizes
    wide = None if window in (20, 9) else (window or 60) + 37 if H % 2 == 0 else 17
    layers = [S.layer(S.attn(H, d, kv=G, vdim=dv, rot=rot, mask=window, scale=5.0 / math.sqrt(d)), None),
              S.layer(S.attn(2 * G, d, kv=G, vdim=dv, rot=rot, mask=wide, scale=5.0 / math.sqrt(d), kv_from=0), None)]
    (m, b), w, spec = mixers_of(layers, dtype, 21)
    assert spec[0]["mixer"]["null_scores"] == "l0.mix.sink" and "k" not in spec[1]["mixer"]
    x = inputs(9)
    kept = [dict() for _ in x]
    ref = [[P.windowed_attention(xb.double(), w, f"l{i}.mix.", layers[i]["mixer"], kept[j], i) for j, xb in enumerate(x)] for i in range(2)]
    k, v = stores(m, dtype)
    got = run_in_portions([m, b], [(k, v, True), (k, v, False)], x, PORTIONS, dtype, LENS)
    for i in range(2):
        for j in range(len(LENS)):
            close(got[i][j], ref[i][j], dtype, f"attention {sizes}, run {i}, sequence {j}", roundings=7.0 if dtype == "bfloat16" else 6.0)


@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_chunked_attention(sizes, dtype):
    H, G, d, dv, rot, chunk = sizes
    layers = [S.layer(S.parallel(S.heads(H, d, kv=G, vdim=dv, rot=rot, mask=chunk, scale=5.0 / math.sqrt(d)), 8, 4, 2, 2), None)]
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, layers)
    spec = _lib.describe_model(c, dtype)["spec"]["layers"][0]["mixer"]["mixers"][0]
    w = {k: v for k, v in S.random_weights(c, 5).items() if ".left." in k and not k.endswith(".out")}
    m = part("mixer", spec, dtype, 1024)
    m.load(w)
    wd = {k: v.double() for k, v in w.items()}
    x = inputs(10)
    k, v = stores(m, dtype)
    got = run_in_portions([m], [(k, v, True)], x, PORTIONS, dtype, LENS)
    for j in range(len(LENS)):
        ref = P.chunked_attention(x[j].double(), wd, "l0.mix.left.", layers[0]["mixer"]["left"])
        close(got[0][j], ref, dtype, f"chunks {sizes}, sequence {j}", roundings=7.0 if dtype == "bfloat16" else 6.0)


@pytest.mark.parametrize("sizes", [(6, 1, 64, 64), (2, 2, 64, 128), (4, 2, 128, 128), (3, 1, 80, 48), (2, 1, 32, 32), (3, 3, 10, 14)])
@pytest.mark.parametrize("kind", ["window", "chunk"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_planted_key_is_seen_up_to_the_edge(sizes, kind, dtype):
    """One key that stands out by far, at a page's first and last place and elsewhere: the last query that sees it gives its value, the
    first that does not gives something else entirely.  Prompts, and single tokens on either side of the edge."""
    H, G, d, dv = sizes
    for size, at in ((9, 63), (64, 64), (64, 10), (100, 127), (70, 70), (128, 1)):
        T = at + size + 4 if kind == "window" else (at // size + 1) * size + 4
        edge = at + size if kind == "window" else (at // size + 1) * size          # the first query that does not see it
        mix = S.heads(H, d, kv=G, vdim=dv, mask=size, scale=1.0)
        layers = [S.layer(dict(type="attention", mixer=mix) if kind == "window" else S.parallel(mix, 8, 4, 2, 2), None)]
        from libllm_b200 import _lib
        c = S.config(64, WIDTH, EPS, layers)
        spec = _lib.describe_model(c, dtype)["spec"]["layers"][0]["mixer"]
        spec = spec if kind == "window" else spec["mixers"][0]
        p = "l0.mix." if kind == "window" else "l0.mix.left."
        w = {k: v for k, v in S.random_weights(c, 3).items() if k.startswith(p) and not k.endswith(".out")}
        u = torch.zeros(d)
        u[3] = 4.0
        # every input has 1 in its first channel, which makes the queries; the planted one has 1 in its second, which makes its key
        w[p + "q"] = torch.zeros_like(w[p + "q"])
        w[p + "q"][:, 0] = u.repeat(H)
        w[p + "k"] = torch.zeros_like(w[p + "k"])
        w[p + "k"][:, 1] = u.repeat(G)
        if kind == "window":
            w[p + "q.b"] *= 0
            w[p + "k.b"] *= 0
        m = part("mixer", spec, dtype, 1024)
        m.load(w)
        wd = {k: v.double() for k, v in w.items()}
        x = inputs(40 + size, [T])[0]
        x[:, 0], x[:, 1] = 1.0, 0.0
        x[at, 1] = 1.0
        run = lambda h: P.windowed_attention(h, wd, p, mix, {}, 0) if kind == "window" else P.chunked_attention(h, wd, p, mix)
        ref = run(x.double())
        plain = x.clone()
        plain[at] = inputs(41, [1])[0][0]
        plain[at, 0], plain[at, 1] = 1.0, 0.0
        moved = (run(plain.double()) - ref).abs().max(-1).values
        assert float(moved[at:edge].min()) > 0.2 and float(moved[edge:].max()) < 1e-12
        k, v = stores(m, dtype)
        for portions in ([[T]], [[edge - 2]] + [[1]] * (T - edge + 2), [[at], [2], [T - at - 2]]):
            if any(q[0] <= 0 for q in portions):
                continue
            got = run_in_portions([m], [(k, v, True)], [x], portions, dtype, [T])[0][0]
            close(got, ref, dtype, f"{kind} {size}, key at {at}, {sizes} cut as {portions[:2]}", roundings=3.0)


@pytest.mark.parametrize("sizes", [(4, 2, 64, 64), (2, 1, 128, 128), (3, 3, 80, 80), (2, 2, 64, 128), (3, 1, 10, 14)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_takes_its_share(sizes, dtype):
    """Sinks far above every score (next to nothing is left), far below (they count for nothing) and beside them, head by head."""
    H, G, d, dv = sizes
    layers = [S.layer(S.attn(H, d, kv=G, vdim=dv, mask=90, scale=0.5 / math.sqrt(d)), None)]

    def sharpen(w):
        w["l0.mix.sink"] = torch.tensor([20.0, -60.0, 3.0, 0.0])[:H].clone()

    (m,), w, _ = mixers_of(layers, dtype, 31, sharpen)
    x = inputs(12)
    k, v = stores(m, dtype)
    got = run_in_portions([m], [(k, v, True)], x, PORTIONS, dtype, LENS)
    for j in range(len(LENS)):
        ref = P.windowed_attention(x[j].double(), w, "l0.mix.", layers[0]["mixer"], {}, 0)
        close(got[0][j], ref, dtype, f"sinks {sizes}, sequence {j}", roundings=3.0)
    # and they do matter: without them the first head's result would be a thousand times as large
    bare = dict(w)
    bare["l0.mix.sink"] = torch.full((H,), -1e9, dtype=torch.float64)
    bare["l0.mix.o"] = w["l0.mix.o"] * (torch.arange(H * dv) < dv)
    with_sink = P.windowed_attention(x[0].double(), dict(bare, **{"l0.mix.sink": w["l0.mix.sink"]}), "l0.mix.", layers[0]["mixer"], {}, 0)
    without = P.windowed_attention(x[0].double(), bare, "l0.mix.", layers[0]["mixer"], {}, 0)
    assert float(with_sink.abs().mean() / without.abs().mean()) < 1e-3


# heads, unrotated, rotated, latent, values, window
LATENT = [(4, 64, 16, 64, 80, 65), (3, 16, 8, 24, 8, 17), (2, 128, 64, 128, 128, 150), (5, 24, 0, 128, 32, 128), (5, 6, 10, 18, 14, None),
          (33, 16, 8, 32, 16, 100), (2, 32, 32, 512, 64, 9), (4, 64, 64, 256, 64, None)]


@pytest.mark.parametrize("sizes", LATENT)
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_with_sinks_and_gates(sizes, dtype):
    """Prompts from the first token (materialised heads), portions and single tokens (all heads over the cached rows), two runs of
    keys joined; sinks head by head from nothing to all."""
    H, d, r, R, dv, window = sizes
    layers = [S.layer(S.latent(H, d, r, R, vdim=dv, mask=window, scale=5.0 / math.sqrt(d + r)), None)]

    def sharpen(w):
        w["l0.mix.sink"] = torch.linspace(-8, 8, H)

    (m,), w, spec = mixers_of(layers, dtype, 22, sharpen)
    assert spec[0]["mixer"]["head_gate"] == "l0.mix.g"
    x = inputs(13)
    k, _ = stores(m, dtype)
    got = run_in_portions([m], [(k, None, True)], x, PORTIONS, dtype, LENS)
    for j in range(len(LENS)):
        ref = P.latent_attention(x[j].double(), w, "l0.mix.", layers[0]["mixer"], EPS)
        close(got[0][j], ref, dtype, f"latent {sizes}, sequence {j}", roundings=7.0 if dtype == "bfloat16" else 6.0)


# ---------------------------------------------------------------- the selective scan
# inner, states, rank, taps: every number of lanes, sizes with and without whole pieces, one tap and eight
SCANS = [(40, 6, 5, 3), (160, 24, 12, 4), (64, 16, 8, 4), (30, 5, 3, 1), (48, 130, 40, 8), (72, 48, 17, 5), (33, 100, 1, 2), (20, 256, 7, 6),
         (256, 32, 64, 4), (8, 1, 2, 2)]


@pytest.mark.parametrize("sizes", SCANS)
def test_selective_scan(sizes):
    """Prompts, portions and single tokens in slots that are used again, one sequence cut every way."""
    layers = [S.layer(S.parallel(S.heads(1, 8), *sizes), None)]
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, layers)
    spec = _lib.describe_model(c, "float32")["spec"]["layers"][0]["mixer"]["mixers"][1]
    assert spec["kind"] == "selective_scan"
    w = {k: v for k, v in S.random_weights(c, 6).items() if ".right." in k and not k.endswith(".out")}
    wd = {k: v.double() for k, v in w.items()}
    check_mixer(spec, w, lambda h: P.selective_mixer(h, wd, "l0.mix.right.", layers[0]["mixer"]["right"]), 14, f"selective scan {sizes}")


def test_a_state_lasts_and_a_state_is_forgotten():
    """Step sizes from next to nothing (a token of the start still counts hundreds of tokens later) to so large that everything before
    is forgotten at once."""
    layers = [S.layer(S.parallel(S.heads(1, 8), 32, 16, 4, 4), None)]
    from libllm_b200 import _lib
    c = S.config(64, WIDTH, EPS, layers)
    spec = _lib.describe_model(c, "float32")["spec"]["layers"][0]["mixer"]["mixers"][1]
    w = {k: v for k, v in S.random_weights(c, 8).items() if ".right." in k and not k.endswith(".out")}
    w["l0.mix.right.dt.b"] = torch.linspace(-9, 30, 32)
    w["l0.mix.right.A_log"] = torch.linspace(-6, 3, 16).repeat(32, 1)
    wd = {k: v.double() for k, v in w.items()}
    run = lambda h: P.selective_mixer(h, wd, "l0.mix.right.", layers[0]["mixer"]["right"])
    x = inputs(15, [320])[0]
    other = x.clone()
    other[0] += 3.0
    assert float((run(other.double()) - run(x.double()))[300:].abs().max()) > 1e-2
    for dtype in DTYPES:
        r = Runner(built(spec, w, dtype), dtype)
        for portions in ([[320]], [[17]] + [[1]] * 100 + [[203]]):
            for t in r.keep:
                t.zero_()
            for xs in (x, other):
                for t in r.keep:
                    t.zero_()
                got = r.run([xs], portions, [320], slots=(2,))[0]
                close(got, run(xs.double()), dtype, f"cut as {portions[:2]}", roundings=4.0 if dtype == "float32" else 8.0)


# ---------------------------------------------------------------- experts
def routed(experts, identity, top, width, ff, shared, dtype, seed, correction=None):
    from libllm_b200 import _lib
    c = S.config(64, width, EPS, [S.layer(S.attn(1, 8), S.moe(experts, top, ff, 0.8, identity=identity, shared=shared))])
    spec = _lib.describe_model(c, dtype)["spec"]["layers"][0]["ff"]
    w = {k: v for k, v in S.random_weights(c, seed).items() if k.startswith("l0.mlp.")}
    if correction is not None:
        w["l0.mlp.correction"] = correction
    m = part("feed_forward", spec, dtype)
    m.load(w)
    return m, {k: v.double() for k, v in w.items()}, c["layers"][0]["mlp"]


@pytest.mark.parametrize("sizes", [(8, 3, 3, 64, 32, (40, 1.1)), (5, 1, 1, 72, 24, None), (6, 2, 2, 54, 20, (36, 0.7)), (16, 4, 4, 128, 64, (128, 1.5)),
                                   (2, 6, 5, 56, 16, (24, 2.0)), (4, 0, 2, 64, 40, (32, 1.0))])
@pytest.mark.parametrize("T", [1, 7, 130, 700])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_among_identity_experts(sizes, T, dtype):
    experts, identity, top, width, ff, shared = sizes
    m, w, f = routed(experts, identity, top, width, ff, shared, dtype, 40 + experts)
    x = bf(torch.randn(T, width, generator=torch.Generator().manual_seed(T)))
    xs = x.to(DT[dtype]).to(DEV)
    got = summed(m.forward(dict(step=Step([T], [0]).json, x=act(xs)))["out"]).cpu()
    margins = []
    ref = P.experts(x.double(), w, "l0.mlp.", f, margins)
    sure = margins[0] > 1e-5           # a closer call is no test (the input is exact in both types, and so is the router's product)
    assert int(sure.sum()) >= 0.9 * T
    close(got[sure], ref[sure], dtype, f"experts {sizes}, {T} tokens", roundings=1.0 if dtype == "bfloat16" else 2.0)


@pytest.mark.parametrize("identity_alone", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_all_choices_are_identity_or_none_is(identity_alone, dtype):
    experts, identity, top, width, ff = 4, 4, 3, 64, 24
    correction = torch.cat([torch.zeros(4), torch.ones(4)]) * (9.0 if identity_alone else -9.0)
    m, w, f = routed(experts, identity, top, width, ff, None, dtype, 50, correction)
    x = bf(torch.randn(33, width, generator=torch.Generator().manual_seed(2)))
    xs = x.to(DT[dtype]).to(DEV)
    got = summed(m.forward(dict(step=Step([33], [0]).json, x=act(xs)))["out"]).cpu()
    margins = []
    ref = P.experts(x.double(), w, "l0.mlp.", f, margins)
    if identity_alone:
        assert float((ref - x.double()).abs().max()) < 1e-12              # the weights add up to one
        close(got, ref, "float32", "identity experts alone")             # no product, no rounding
    else:
        sure = margins[0] > 1e-5
        close(got[sure], ref[sure], dtype, "experts alone")


@pytest.mark.parametrize("width,ff", [(64, 40), (128, 256), (54, 22)])
@pytest.mark.parametrize("T", [1, 20, 60, 200, 1100])
@pytest.mark.parametrize("dtype", DTYPES)
def test_bounded_unit_alone(width, ff, T, dtype):
    """The unit with its bounds active, fused into the product (few tokens, and prompts long enough) or behind it."""
    w = {n: bf(torch.randn(*s, generator=torch.Generator().manual_seed(i)) * 1.5 / math.sqrt(s[1]))
         for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))}
    m = part("feed_forward", dict(kind="clamped_glu", hidden=width, intermediate=ff, limit=0.9, slope=1.702, up_shift=1.0, gate="gate", up="up",
                                  down="down"), dtype)
    m.load(w)
    x = bf(torch.randn(T, width, generator=torch.Generator().manual_seed(T)))
    xs = x.to(DT[dtype]).to(DEV)
    got = summed(m.forward(dict(step=Step([T], [0]).json, x=act(xs)))["out"]).cpu()
    close(got, P.bounded_unit(x.double(), {k: v.double() for k, v in w.items()}, "", 0.9), dtype, "bounded unit")
