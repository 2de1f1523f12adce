"""Fomodra's configuration, its description as parts, borrowed caches, the faults it names: what needs no GPU.  Also the plain
implementation's small functions by hand, and the cache's books for a window that is kept for a borrower."""
import copy
import math

import pytest
import torch

import fomodra_helpers as S
import plain_fomodra as P

F64 = torch.float64


def describe(c, dtype="bfloat16"):
    from libllm_b200 import _lib
    return _lib.describe_model(c, dtype)


@pytest.mark.parametrize("name", sorted(S.CONFIGS))
def test_tensors_asked_for_are_the_designs_names_and_shapes(name):
    c = S.CONFIGS[name]
    d = describe(c)
    assert {t["name"]: t["shape"] for t in d["tensor_needs"]} == S.tensor_shapes(c)
    roles = {t["name"]: t["role"] for t in d["tensor_needs"]}
    assert roles["embed"] == roles["head"] == "matrix"
    for n, r in roles.items():
        end = n.split(".")[-1]
        if end in ("norm", "norm1", "norm1b", "norm2", "norm2b", "out", "sink", "b", "correction", "A_log", "D", "conv"):
            assert r == "vector", n                                        # 32-bit, whatever the engine's type
    assert d["capturable"]


@pytest.mark.parametrize("name", sorted(S.CONFIGS))
def test_order_of_runs_and_whose_cache_each_reads(name):
    c = S.CONFIGS[name]
    sched = describe(c)["spec"]["schedule"]
    assert [e["layer"] for e in sched] == list(range(len(c["layers"])))
    assert [e["cache_from"] for e in sched] == [L["mixer"].get("kv_from") for L in c["layers"]]


def test_every_constant_reaches_its_part():
    c = S.CONFIGS["K1"]
    spec = describe(c)["spec"]
    assert spec["token_pairs"] == dict(table="bigram", buckets=53, mul_prev=13, mul_cur=7)
    assert (spec["token_table"], spec["token_table_width"]) == ("side.embed", 50)
    assert (spec["embedding"], spec["head"], spec["streams"]) == ("embed", "head", 1)
    assert spec["final_norm"] == dict(kind="rmsnorm", size=64, eps=1e-6, weight="final.norm")
    L = spec["layers"]
    for i, b in enumerate(L):
        assert b["kind"] == "prenorm" and b["mixer_norm"]["weight"] == f"l{i}.norm1" and b["mixer_post"] == dict(weight=f"l{i}.norm1b", eps=1e-6)
        assert b["side"] == dict(dim=10, offset=10 * i, eps=1e-6, gate=f"l{i}.side.gate", proj=f"l{i}.side.proj", norm=f"l{i}.side.norm")
    assert L[0]["ff_norm"]["weight"] == "l0.norm2" and L[0]["ff_post"]["weight"] == "l0.norm2b"
    assert L[1]["ff"] is None and L[1]["ff_norm"] is None and "ff_post" not in L[1]
    a = L[0]["mixer"]
    assert (a["kind"], a["n_heads"], a["n_kv_heads"], a["head_dim"], a["v_head_dim"], a["window"], a["bias"], a["null_scores"]) == \
        ("attention", 6, 2, 16, 16, 24, True, "l0.mix.sink")
    assert a["k_bias"] == "l0.mix.k.b" and a["q_bias"] == "l0.mix.q.b" and abs(a["scale"] - 1.7 / 4) < 1e-15
    assert a["position"] == dict(kind="rope", head_dim=16, rotary_dim=8, theta=5e4, pairing="half", scaling=None)
    assert a["cache_window"] == 70                                         # the borrower looks farther back than the lender
    b = L[4]["mixer"]
    assert b["window"] == 70 and not {"k", "v", "k_bias", "v_bias", "cache_window"} & set(b) and b["q_bias"] == "l4.mix.q.b"
    s = L[1]["mixer"]
    assert s["kind"] == "sum" and [m["kind"] for m in s["mixers"]] == ["attention", "selective_scan"]
    assert s["norms"] == dict(hidden=64, eps=1e-6, scale=0.5, weights=["l1.mix.left.out", "l1.mix.right.out"])
    left, right = s["mixers"]
    assert left["block"] == 20 and "window" not in left and "bias" not in left and "null_scores" not in left and left["v_head_dim"] == 32
    assert left["position"]["scaling"] == dict(rope_type="llama3", factor=4.0, original_max_position_embeddings=64, low_freq_factor=1.0,
                                               high_freq_factor=4.0)
    assert (right["inner"], right["state"], right["dt_rank"], right["taps"]) == (40, 6, 5, 3)
    assert right["a_log"] == "l1.mix.right.A_log" and right["skip"] == "l1.mix.right.D" and right["conv_bias"] == "l1.mix.right.conv.b"
    m = L[3]["mixer"]
    assert (m["kind"], m["n_heads"], m["head_dim"], m["rot_dim"], m["v_head_dim"], m["kv_rank"], m["window"]) == \
        ("latent_attention", 3, 16, 8, 8, 24, 17)
    assert m["q"] == "l3.mix.q" and m["null_scores"] == "l3.mix.sink" and m["head_gate"] == "l3.mix.g" and "q_down" not in m
    f = L[0]["ff"]
    assert (f["kind"], f["experts"], f["identity"], f["top"], f["score"], f["renormalize"], f["norm_eps"], f["weight_on"]) == \
        ("moe", 6, 2, 2, "softmax", True, 1e-20, "output")
    assert f["correction"] == "l0.mlp.correction" and "groups" not in f
    assert f["expert"] == dict(intermediate=24, activation="bounded_glu", limit=1.0, slope=1.702, up_shift=1.0, gate="l0.mlp.e{}.gate",
                               up="l0.mlp.e{}.up", down="l0.mlp.e{}.down")
    assert (f["shared"]["kind"], f["shared"]["intermediate"], f["shared"]["limit"], f["shared"]["slope"], f["shared"]["up_shift"]) == \
        ("clamped_glu", 40, 1.5, 1.702, 1.0)
    # what a configuration leaves out
    k2 = describe(S.CONFIGS["K2"])["spec"]
    assert "token_pairs" not in k2 and "token_table" not in k2 and all("side" not in b for b in k2["layers"])
    assert k2["layers"][0]["mixer"]["position"] is None and "window" not in k2["layers"][0]["mixer"] and k2["layers"][0]["ff"]["identity"] == 0
    # a borrower that sees everything: the lender's cache keeps everything
    assert describe(S.CONFIGS["K3"])["spec"]["layers"][0]["mixer"]["cache_window"] == 0
    assert describe(S.CONFIGS["K5"])["spec"]["layers"][3]["mixer"]["cache_window"] == 150


def test_faults_are_named():
    from libllm_b200.errors import ConfigError
    base = S.CONFIGS["K1"]

    def broken(change, match):
        c = copy.deepcopy(base)
        change(c)
        with pytest.raises(ConfigError, match=match):
            describe(c)

    broken(lambda c: c["layers"][0].update(type="conv"), "not known")
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of 'kv_heads'")
    broken(lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple of 'kv_heads'")
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "'dims'")
    broken(lambda c: c["layers"][1]["mixer"].pop("right"), "right")
    broken(lambda c: c["layers"][1]["mixer"]["right"].pop("state"), "state")
    broken(lambda c: c["layers"][3]["mixer"]["rot"].update(dims=4), "rot_dim")
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "'top' exceeds")
    broken(lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit")
    broken(lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff")
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=4), "earlier layer")
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=1), "keys and values of its own")
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=2), "differs")
    broken(lambda c: c["layers"][4]["mixer"].update(vdim=8), "'vdim' differs")
    broken(lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets")
    broken(lambda c: c["token_side"].pop("dim"), "dim")
    broken(lambda c: c.pop("norm"), "norm")


def test_parts_refuse_what_does_not_go_together():
    from libllm_b200.errors import LlmError
    from libllm_b200.parts import PartHandle
    spec = describe(S.CONFIGS["K1"])["spec"]["layers"]
    both = copy.deepcopy(spec[0])
    both["mixer_scale"] = "s"
    with pytest.raises(LlmError, match="a scale or a norm"):
        PartHandle("block", both)
    three = copy.deepcopy(spec[1]["mixer"])
    three["mixers"].append(three["mixers"][1])
    three["norms"]["weights"].append("x")
    with pytest.raises(LlmError, match="two mixers"):
        PartHandle("mixer", three)
    narrow = copy.deepcopy(spec[0]["mixer"])
    narrow["cache_window"] = 5
    with pytest.raises(LlmError, match="cache_window"):
        PartHandle("mixer", narrow)
    plain = copy.deepcopy(spec[0]["ff"])
    plain["expert"].pop("gate")
    with pytest.raises(LlmError, match="gated experts"):
        PartHandle("feed_forward", plain)


def test_what_each_run_keeps():
    from libllm_b200.parts import PartHandle
    spec = describe(S.CONFIGS["K1"], "float32")["spec"]["layers"]
    cache = lambda i: PartHandle("mixer", spec[i]["mixer"], "float32").description["cache"]
    assert (cache(0)["kind"], cache(0)["window"], cache(0)["k_dim"], cache(0)["v_dim"]) == ("window", 70, 16, 16)
    assert (cache(1)["kind"], cache(1)["block"], cache(1)["v_dim"]) == ("block", 20, 32)
    assert (cache(3)["kind"], cache(3)["window"], cache(3)["k_dim"], cache(3)["v_dim"]) == ("window", 17, 32, 0)
    full = PartHandle("mixer", describe(S.CONFIGS["K3"])["spec"]["layers"][0]["mixer"]).description["cache"]
    assert full["kind"] == "full"
    state = PartHandle("mixer", spec[1]["mixer"], "float32").description["state"]
    assert [(s["name"], s["shape"], s["dtype"]) for s in state] == [("1:selective_scan.S", [40, 6], "float32"),
                                                                  ("1:selective_scan.inputs", [2, 40], "float32")]


# ---------------------------------------------------------------- the plain functions by hand
def test_plain_rows_of_token_pairs():
    c = dict(embedding=dict(bigram=dict(buckets=10, mul_prev=3, mul_cur=4)))
    w = dict(embed=torch.zeros(9, 1, dtype=F64), bigram=torch.arange(11, dtype=F64)[:, None])
    assert P.token_rows(c, w, [5, 2, 8])[:, 0].tolist() == [10.0, (15 + 8) % 10, (6 + 32) % 10]


def test_plain_masks():
    assert P.visible(4, window=2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False],
                                               [False, False, True, True]]
    assert P.visible(4, chunk=3).tolist() == [[True, False, False, False], [True, True, False, False], [True, True, True, False],
                                              [False, False, False, True]]


def test_plain_softmax_with_a_sink():
    s, one = torch.zeros(1, 2, dtype=F64), torch.ones(1, 2, dtype=torch.bool)
    assert torch.allclose(P.softmax_with_sink(s, one, torch.tensor(math.log(2.0), dtype=F64)), torch.full((1, 2), 0.25, dtype=F64))
    assert torch.allclose(P.softmax_with_sink(s, one, None), torch.full((1, 2), 0.5, dtype=F64))


def test_plain_frequencies_by_wavelength():
    rot = dict(dims=2, base=10.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=0))
    wave = 2 * math.pi                                                     # of the one pair: frequency 1
    for original, want in ((wave * 5, 1.0), (wave * 0.5, 0.25), (wave * 2.5, 0.5 * 0.25 + 0.5)):
        rot["scaling"]["original"] = original
        assert abs(float(P.frequencies(rot)[0]) - want) < 1e-12


def test_plain_selective_scan():
    one = lambda *v: torch.tensor(v, dtype=F64)[:, None]
    A, D = torch.tensor([[-math.log(2.0)]], dtype=F64), torch.tensor([10.0], dtype=F64)
    y = P.selective_scan(one(1, 2), one(1, 3), A, one(5, 7), one(1, 1), D)
    assert torch.allclose(y[:, 0], torch.tensor([5.0 + 10, 5 / 8 + 3 * 2 * 7 + 20], dtype=F64))


def test_plain_choice_with_identity_experts():
    h = torch.eye(2, dtype=F64)[:1]
    w = {"router": torch.zeros(3, 2, dtype=F64), "correction": torch.tensor([0.0, 0.0, 5.0], dtype=F64)}
    w["router"][:, 0] = torch.tensor([2.0, 1.0, -3.0])
    chosen, weight, _ = P.route(h, w, "", dict(experts=2, identity=1, top=2))
    s = torch.softmax(w["router"][:, 0], 0)
    assert chosen.tolist() == [[2, 0]]                                     # the correction turns the choice, not the weights
    assert torch.allclose(weight[0], s[[2, 0]] / (s[2] + s[0]))


def test_plain_bounded_unit():
    w = dict(gate=torch.eye(2, dtype=F64), up=torch.eye(2, dtype=F64), down=torch.eye(2, dtype=F64))
    y = P.bounded_unit(torch.tensor([[3.0, -4.0]], dtype=F64), w, "", 1.5)
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert torch.allclose(y[0], torch.tensor([f(1.5, 1.5), f(-4.0, -1.5)], dtype=F64))
