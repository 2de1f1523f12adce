"""The Fomodra decoder through the engine (its step function, cache and state manager, scheduler) against the plain
implementation, in float32 and bfloat16, for every way of cutting the work: whole prompts, prompts then single tokens,
portions of prompts down to one token, unequal batches, pages and slots used again, long decoding across page borders and
window edges, the first tokens, other sizes, and greedy generation."""
import copy
import json
import os
import subprocess

import pytest
import torch

import plain_fomodra as P
import fomodra_helpers as S
from libllm_b200.engine import GREEDY, StepItem
from replay import replay_batch

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
NAMES = sorted(S.CONFIGS)
_engines, _refs = {}, {}


def setup(name, dtype, max_tokens=4096, **kw):
    from libllm_b200.engine import Engine
    key = (name, dtype, max_tokens, tuple(sorted(kw.items())))
    if key not in _engines:
        c = S.CONFIGS[name] if dtype == "float32" else S.every_expert(S.CONFIGS[name])
        w = S.random_weights(c, seed=ord(name[-1]))
        _engines[key] = (Engine.from_tensors(c, w, dtype=dtype, max_tokens=max_tokens, **kw), c, w)
    return _engines[key]


def plain(c, w, toks, dtype):
    """-> logits, and per position the smallest margin of any router's choice (float32) or the weight of a rounding (bfloat16)"""
    key = (json.dumps(c), tuple(toks), dtype, float(sum(v.sum() for v in w.values())))
    if key not in _refs:
        margins = []
        logits = P.forward(c, w, toks, margins=margins)
        if dtype == "float32":
            _refs[key] = (logits, torch.stack(margins).min(0).values if margins else None, None)
        else:
            _refs[key] = (logits, None, S.noise(P.forward, c, w, toks, logits))
    return _refs[key]


def compare(got, c, w, toks, dtype, what, rows=None):
    ref, margin, rounding = plain(c, w, toks, dtype)
    if rows is not None:
        ref, margin, rounding = ref[rows], margin[rows] if margin is not None else None, rounding[rows] if rounding is not None else None
    S.check_rows(got, ref, dtype, what, margin, rounding)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(name, dtype):
    """Lengths from one token on, around the convolutions' taps, the scan's groups (8 and 16), the masks (9 to 150) and the page
    border (64)."""
    engine, c, w = setup(name, dtype)
    toks = S.tokens(c, 203, 0)
    for n in [1, 2, 3, 4, 8, 9, 10, 15, 16, 17, 25, 33, 63, 64, 65, 101, 151, 203]:
        got = replay_batch(engine, [("r", toks[:n], n)])["r"]
        compare(got, c, w, toks, dtype, f"{name} whole {n}", rows=slice(0, n))   # causal: a shorter prompt's logits come first
    assert engine.pages_in_use() == [0] * len(engine.pages_in_use())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_models_cut_after_every_layer(name, dtype):
    """Models cut after 1, 2, .. layers give the logits of the plain model cut at the same place: a fault shows at the first layer
    that has it."""
    from libllm_b200.engine import Engine
    c_full = S.CONFIGS[name] if dtype == "float32" else S.every_expert(S.CONFIGS[name])
    w_full = S.random_weights(c_full, seed=3)
    toks = S.tokens(c_full, 90, 4)
    for n in range(1, len(c_full["layers"])):
        c = copy.deepcopy(c_full)
        c["layers"] = c["layers"][:n]
        keep = tuple(f"l{i}." for i in range(n))
        w = {k: v for k, v in w_full.items() if not (k.startswith("l") and k[1].isdigit()) or k.startswith(keep)}
        if "side.embed" in w:
            w["side.embed"] = w["side.embed"][:, :n * c["token_side"]["dim"]].contiguous()
        engine = Engine.from_tensors(c, w, dtype=dtype, max_tokens=256)
        got = replay_batch(engine, [("r", toks, 60)])["r"]
        compare(got, c, w, toks, dtype, f"{name}: the first {n} layers")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_single_tokens_agrees_with_the_whole_prompt(name, dtype):
    """The same request as one prompt and as a prompt followed by single tokens, which pass page borders and carry every
    window and state over decoded tokens; also from a one-token prompt on."""
    engine, c, w = setup(name, dtype)
    for i, (n, n_prompt) in enumerate([(180, 100), (75, 35), (48, 1)]):
        toks = S.tokens(c, n, 20 + i)
        got = replay_batch(engine, [("r", toks, n_prompt)])["r"]
        compare(got, c, w, toks, dtype, f"{name} {n_prompt} + {n - n_prompt} single tokens")
        if dtype == "float32":
            whole = replay_batch(engine, [("r", toks, n)])["r"]
            S.check_rows(got, whole, dtype, f"{name}: decoding against the whole prompt", plain(c, w, toks, dtype)[1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_a_prompt(name, dtype):
    """A prompt brought in portions of several sizes, down to two tokens and one: a portion's first tokens look back
    into cached rows through every window and chunk, into the convolutions' last inputs, the token before and every state."""
    engine, c, w = setup(name, dtype)
    toks = S.tokens(c, 212, 31)
    for sizes in ([64, 64, 64, 20], [2] * 20 + [57, 3, 100, 12], [7, 1, 42, 50, 2, 26, 70, 14], [1, 1, 1, 2, 1, 3, 203]):
        assert sum(sizes) == len(toks)
        slot = engine.open_sequence()
        rows, at = [], 0
        for n in sizes:
            rows.append(torch.from_numpy(engine.step([StepItem(slot, toks[at:at + n], list(range(n)))])))
            at += n
        engine.close_sequence(slot)
        compare(torch.cat(rows), c, w, toks, dtype, f"{name} portions {sizes[:4]}...")
    engine.cache_check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_steps(name, dtype):
    """Steps in which some sequences bring portions and others single tokens, each compared with its plain run."""
    engine, c, w = setup(name, dtype)
    lens = [90, 41, 70]
    toks = [S.tokens(c, n, 60 + i) for i, n in enumerate(lens)]
    plan = [[30, 1, 0], [1, 2, 20], [2, 30, 1], [50, 1, 1], [1, 1, 40], [5, 5, 1], [1, 1, 7]]
    assert [sum(p[b] for p in plan) for b in range(3)] == lens
    slots, done, rows = [engine.open_sequence() for _ in lens], [0] * 3, [[], [], []]
    for p in plan:
        live = [b for b in range(3) if p[b]]
        got = torch.from_numpy(engine.step([StepItem(slots[b], toks[b][done[b]:done[b] + p[b]], list(range(p[b]))) for b in live]))
        at = 0
        for b in live:
            rows[b].append(got[at:at + p[b]])
            done[b] += p[b]
            at += p[b]
    for b in range(3):
        engine.close_sequence(slots[b])
        compare(torch.cat(rows[b]), c, w, toks[b], dtype, f"{name} mixed steps, sequence {b}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_against_each_request_alone(name, dtype):
    """Three batches of unequal requests on a cache that holds one batch at a time, so that pages, slots and state are used
    again; shorter requests end earlier; each request against the plain implementation and, in float32, against
    itself alone."""
    prompts, n_dec = [1, 70, 9, 131], 12
    cap = sum((p + n_dec + 4 + 63) // 64 * 64 for p in prompts)
    engine, c, w = setup(name, dtype, max_tokens=cap)
    alone, _, _ = setup(name, dtype)
    for b in range(3):
        reqs = []
        for j, p in enumerate(prompts):
            total = p + n_dec - (j if b % 2 == 0 else 3 - j)
            reqs.append((f"b{b}r{j}", S.tokens(c, total, 100 * b + j), p))
        got = replay_batch(engine, reqs)
        for rid, toks, p in reqs:
            compare(got[rid], c, w, toks, dtype, f"{name} batch {b} {rid}")
            if dtype == "float32" and b == 0:
                single = replay_batch(alone, [(rid, toks, p)])[rid]
                S.check_rows(got[rid], single, dtype, f"{name} {rid}: the batch changes the result", plain(c, w, toks, dtype)[1])
    assert engine.pages_in_use() == [0] * len(engine.pages_in_use())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["K1", "K3", "K4"])
def test_long_decoding(name, dtype):
    """One token a step for 330 steps: pages are taken as the rows grow over five page borders and given back as they
    leave the windows."""
    engine, c, w = setup(name, dtype)
    toks = S.tokens(c, 330, 77)
    got = replay_batch(engine, [("r", toks, 2)])["r"]
    compare(got, c, w, toks, dtype, f"{name} long decoding")


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_beside_a_long_neighbour(dtype):
    engine, c, w = setup("K1", dtype)
    short, long_ = S.tokens(c, 3, 5), S.tokens(c, 90, 6)
    both = replay_batch(engine, [("l", long_, 60), ("s", short, 1)])
    compare(both["s"], c, w, short, dtype, "first tokens beside a long request")
    compare(both["l"], c, w, long_, dtype, "long neighbour")


@pytest.mark.parametrize("name", NAMES)
def test_a_sequence_starts_from_nothing_whatever_its_slot_held(name):
    """The same request before and after others have used its slot: bit for bit the same logits."""
    engine, c, w = setup(name, "float32")
    toks = S.tokens(c, 40, 8)
    first = replay_batch(engine, [("r", toks, 25)])["r"]
    replay_batch(engine, [("x", S.tokens(c, 90, 9), 80), ("y", S.tokens(c, 33, 10), 20)])
    assert torch.equal(first, replay_batch(engine, [("r", toks, 25)])["r"])


@pytest.mark.parametrize("name", NAMES)
def test_what_the_cache_holds(name):
    """Every layer with keys and values of its own has pages, of its widths; a window or a chunk gives pages back, but for those a
    layer that borrows the keys still sees; a borrower holds none.  The last token is state of the model."""
    engine, c, w = setup(name, "float32")
    n, slot = 330, engine.open_sequence()
    engine.step([StepItem(slot, S.tokens(c, n, 3), [n - 1])])
    info = engine.cache_info()
    owners = [i for i, L in enumerate(c["layers"]) if L["mixer"].get("kv_from") is None]
    assert sorted(r for g in info["groups"] for r in g["runs"]) == owners
    for g in info["groups"]:
        for r in g["runs"]:
            L = c["layers"][r]
            m = L["mixer"]["left"] if L["type"] == "parallel" else L["mixer"]
            size = (m.get("mask") or {}).get("size")
            if L["type"] == "latent_attention":
                assert (g["n_kv_heads"], g["k_dim"], g["v_dim"]) == (1, m["kv_rank"] + m["rot_dim"], 0), g
            else:
                assert (g["n_kv_heads"], g["k_dim"], g["v_dim"]) == (m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])), g
            if L["type"] == "parallel":
                assert g["block"] == size
                first = n // size * size if size else 0
            else:
                reach = [size] + [(o["mixer"].get("mask") or {}).get("size") for o in c["layers"] if o["mixer"].get("kv_from") == r]
                window = None if None in reach else max(reach)
                assert g["window"] == window, g
                first = n - window + 1 if window else 0
            pages = (n + 63) // 64 - first // 64
            assert g["pages_in_use"] in (pages, pages * len(g["runs"])), g
    assert len(info["state"]) == len(c["layers"]) + (1 if c.get("embedding") else 0)
    engine.close_sequence(slot)
    engine.cache_check()
    assert engine.pages_in_use() == [0] * len(engine.pages_in_use())


def test_the_previous_token_is_the_sequences_own():
    """Two sequences in one step, in portions and single tokens, with a slot that another sequence has used: the pair of a token is
    made with the token before it in its own sequence, and a first token has none.  The weights make the pair's row the largest
    part of the stream."""
    from libllm_b200.engine import Engine
    c = S.CONFIGS["K1"]
    w = S.random_weights(c, 4)
    w["bigram"] = w["bigram"] * 4
    engine = Engine.from_tensors(c, w, dtype="float32", max_tokens=1024)
    toks = [S.tokens(c, 20, 300 + i) for i in range(3)]
    replay_batch(engine, [("x", toks[2], 7), ("y", toks[1], 3)])
    plan = [[1, 4], [1, 0], [3, 1], [0, 1], [15, 14]]
    slots, done, rows = [engine.open_sequence() for _ in range(2)], [0, 0], [[], []]
    for p in plan:
        live = [b for b in range(2) if p[b]]
        got = torch.from_numpy(engine.step([StepItem(slots[b], toks[b][done[b]:done[b] + p[b]], list(range(p[b]))) for b in live]))
        at = 0
        for b in live:
            rows[b].append(got[at:at + p[b]])
            done[b] += p[b]
            at += p[b]
    for b in range(2):
        engine.close_sequence(slots[b])
        compare(torch.cat(rows[b]), c, w, toks[b], "float32", f"sequence {b}")


def test_a_borrower_sees_beyond_its_lenders_window():
    """A key that stands out far back: inside the borrower's window, long out of the lender's, after pages between have been given
    back; and just outside the borrower's window.  Prompt and single tokens, both types."""
    from libllm_b200.engine import Engine
    c = S.config(64, 64, 1e-6, [S.layer(S.attn(2, 64, kv=1, rot=(2, 1e6), mask=10), None),
                                S.layer(S.attn(4, 64, kv=1, rot=(2, 1e6), mask=200, kv_from=0, scale=2.0), None)], pairs=(7, 1, 1))
    w = S.random_weights(c, 9)
    # token 5's key is along one direction which every query of the borrower likes, and its value is large
    u = torch.zeros(64)
    u[10] = 1.0
    w["bigram"] *= 0
    w["embed"][:, 0] = 0
    w["embed"][5] *= 0.1
    w["embed"][5, 0] = 6.0
    w["l0.mix.k"] *= 0.05
    w["l0.mix.k"][:, 0] = u * 4
    w["l1.mix.q.b"] = u.repeat(4) * 3
    w["l1.mix.q"] *= 0.1
    toks = [t if t != 5 else 6 for t in S.tokens(c, 330, 2)]
    toks[3] = 5
    ref = P.forward(c, w, toks)
    for at in (202, 203):                                # the last query that sees it, the first that does not
        other = list(toks)
        other[3] = 6
        moved = float((P.forward(c, w, other)[at] - ref[at]).abs().max())
        assert (moved > 0.5) == (at == 202), (at, moved)
    for dtype in DTYPES:
        engine = Engine.from_tensors(c, w, dtype=dtype, max_tokens=512)
        for n_prompt in (330, 150, 203):
            got = replay_batch(engine, [("r", toks, n_prompt)])["r"]
            S.check_rows(got, ref, dtype, f"{n_prompt} tokens of prompt ({dtype})")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["K2", "K3"])
def test_a_step_cut_into_launch_sequences(name, dtype):
    """max_step_tokens below the prompts' lengths: the engine itself cuts inside a prompt."""
    engine, c, w = setup(name, dtype, max_step_tokens=48)
    reqs = [("a", S.tokens(c, 150, 1), 150), ("b", S.tokens(c, 30, 2), 30)]
    got = replay_batch(engine, reqs)
    for rid, toks, _ in reqs:
        compare(got[rid], c, w, toks, dtype, f"cut {rid}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_of_more_tokens_than_the_small_product_takes(dtype):
    """600 tokens in one step: the library products, the sums that ride on them, the wide tiles."""
    engine, c, w = setup("K3", dtype)
    toks = S.tokens(c, 600, 12)
    compare(replay_batch(engine, [("r", toks, 590)])["r"], c, w, toks, dtype, "a prompt of 590 tokens")


@pytest.mark.parametrize("name", NAMES)
def test_the_last_row_alone(name):
    """A prompt of which only some places are wanted (the last layer then runs its feed-forward for those rows
    alone), and a portion of which nothing is wanted (its cache and state still move on)."""
    engine, c, w = setup(name, "float32")
    toks = S.tokens(c, 77, 9)
    slot = engine.open_sequence()
    assert engine.step([StepItem(slot, toks[:40], [])]).shape[0] == 0
    got = torch.from_numpy(engine.step([StepItem(slot, toks[40:], [36, 0])]))
    engine.close_sequence(slot)
    compare(got, c, w, toks, "float32", f"{name} chosen rows", rows=[76, 40])


@pytest.mark.parametrize("name", ["K1", "K3", "K5"])
def test_greedy_generation_through_the_generation_loop(name):
    """engine.generate (scheduler, sampling, stop rule) in float32 against the plain implementation's own greedy
    loop, for prompts of unequal lengths in one call."""
    engine, c, w = setup(name, "float32")
    prompts = [S.tokens(c, n, 50 + n) for n in (5, 23, 1)]
    out = engine.generate(prompts, max_new_tokens=[10, 6, 12], sampling=GREEDY, stop_tokens=[])
    for p, got, n in zip(prompts, out, (10, 6, 12)):
        seq = list(p)
        for _ in range(n):
            logits = P.forward(c, w, seq)[-1]
            top2 = logits.topk(2).values
            if float(top2[0] - top2[1]) < 1e-3:        # a close call is no test of anything
                break
            seq.append(int(logits.argmax()))
        want = seq[len(p):]
        assert got[:len(want)] == want, f"{name}: generated {got}, the plain loop {want}"
        assert len(got) == n


def fomodra_folder(tmp_path, c, seed):
    from helpers import write_safetensors
    w = S.random_weights(c, seed)
    (tmp_path / "config.json").write_text(json.dumps(c))
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    return str(tmp_path), w


def test_the_model_folder_route_names_what_does_not_fit(tmp_path):
    """Weights written as a safetensors file and loaded by folder give the engine that tensors in memory give; an
    unexpected or missing tensor is named, and so is one of the wrong shape."""
    from libllm_b200.engine import Engine
    from libllm_b200.errors import WeightsError
    c = S.CONFIGS["K2"]
    folder, w = fomodra_folder(tmp_path, c, 3)
    engine = Engine.from_folder(folder, dtype="float32", max_tokens=256)
    toks = S.tokens(c, 40, 1)
    compare(replay_batch(engine, [("r", toks, 30)])["r"], c, w, toks, "float32", "from a folder")
    del w["l1.mix.right.A_log"]
    w["l2.mix.k"] = torch.zeros(66, 3)
    with pytest.raises(WeightsError) as e:
        Engine.from_tensors(c, w, dtype="float32", max_tokens=256)
    assert e.value.missing == ["l1.mix.right.A_log"] and e.value.unexpected == ["l2.mix.k"]
    w = S.random_weights(c, 3)
    w["l0.mix.sink"] = torch.ones(c["width"])
    with pytest.raises(WeightsError, match="l0.mix.sink"):
        Engine.from_tensors(c, w, dtype="float32", max_tokens=256)
    # a layer without a feed-forward may have its norms in the files all the same
    w = S.random_weights(c, 3)
    w["l2.norm2"] = torch.ones(c["width"])
    Engine.from_tensors(c, w, dtype="float32", max_tokens=256)


def test_the_command_line_generates_from_a_fomodra_folder(tmp_path):
    """``bin/llm generate`` picks the model by config.json's ``architecture`` and builds what it needs."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    c = S.CONFIGS["K4"]
    folder, w = fomodra_folder(tmp_path, c, 8)
    prompt = S.tokens(c, 7, 800)
    out = subprocess.run([os.path.join(root, "bin", "llm"), "generate", "-m", folder, "--prompt-ids", ",".join(map(str, prompt)),
                          "--max-new-tokens", "4", "--temperature", "0", "--dtype", "float32", "--no-stop"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    got = [int(t) for t in out.stdout.strip().splitlines()[-1].split(",")]
    seq = list(prompt)
    for tok in got:
        logits = P.forward(c, w, seq)[-1]
        top2 = logits.topk(2)
        assert tok == int(top2.indices[0]) or float(top2.values[0] - top2.values[1]) < 1e-3
        seq.append(tok)
    assert len(got) == 4


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_of_a_fomodra_folder(dtype, tmp_path):
    """``bin/trace_run`` on a folder: two unequal requests that start together and go on by single tokens, then a
    third alone that uses their slots and pages again."""
    from test_entry_points_gpu import collect, run_trace, trace_of
    c = S.CONFIGS["K3"] if dtype == "float32" else S.every_expert(S.CONFIGS["K3"])
    folder, w = fomodra_folder(tmp_path, c, 9)
    first = [("a", S.tokens(c, 120, 1), 101), ("b", S.tokens(c, 40, 2), 7)]
    steps = trace_of(first)
    steps += trace_of([("c", S.tokens(c, 70, 3), 66)], first_step=len(steps))
    out_dir = str(tmp_path / "out")
    run_trace(folder, dtype, steps, out_dir, max_tokens=256)
    got = collect(steps, out_dir, c["vocab"])
    for rid, toks, _ in first + [("c", S.tokens(c, 70, 3), 66)]:
        compare(got[rid], c, w, toks, dtype, f"trace {rid}")


def test_a_drawn_model_generates():
    """Random weights drawn on the device (the mode the throughput figures use) give finite logits and tokens in range."""
    from libllm_b200 import Model
    c = S.CONFIGS["K3"]
    model = Model.from_random(c, seed=1, dtype="bfloat16", max_tokens=1024, max_seq_len=512)
    out = model.generate([S.tokens(c, 20, 1)], max_new_tokens=8, temperature=0.0, top_k=1, top_p=1.0, seed=0, stop_token_ids=[])
    assert len(out[0]) == 8 and all(0 <= t < c["vocab"] for t in out[0])
