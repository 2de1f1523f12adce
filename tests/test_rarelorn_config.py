"""Rarelorn's configuration, its description as parts, the order of its runs and what a pass adds, the faults it names: what
needs no GPU.  Also the plain implementation's small functions by hand."""
import copy
import math

import pytest
import torch

import plain_rarelorn as P
import rarelorn_helpers as S


def describe(c, dtype="bfloat16"):
    from libllm_b200 import _lib
    return _lib.describe_model(c, dtype)


@pytest.mark.parametrize("name", sorted(S.CONFIGS))
def test_tensors_asked_for_are_the_designs_names_and_shapes(name):
    c = S.CONFIGS[name]
    d = describe(c)
    need = {t["name"]: t["shape"] for t in d["tensor_needs"]}
    free = {n for n, s in need.items() if -1 in s}
    assert free == {n for n in need if n.endswith("right.w1") or n.endswith("right.w2")}     # the rank is the stored tensor's
    want = S.tensor_shapes(c)
    assert {n: want[n] if n in free else s for n, s in need.items()} == want
    roles = {t["name"]: t["role"] for t in d["tensor_needs"]}
    assert roles["l0.norm1"] == roles["final.norm"] == "vector" and roles["embed"] == roles["head"] == "matrix"
    for n, r in roles.items():
        end = n.split(".")[-1]
        if end in ("dt_bias", "A_log", "temp", "pb", "u", "w0", "w2", "conv", "step") or ".mu." in n:
            assert r == "vector", n                                        # 32-bit, whatever the engine's type
    assert d["capturable"]


@pytest.mark.parametrize("name", sorted(S.CONFIGS))
def test_order_of_runs_and_what_each_pass_adds(name):
    c = S.CONFIGS[name]
    sched = describe(c)["spec"]["schedule"]
    runs = P.order_of_runs(c)
    assert [e["layer"] for e in sched] == [i for i, _ in runs]
    for e, (_, t) in zip(sched, runs):
        assert e["cache_from"] is None and e["input_mix"] is None
        assert e.get("add_tokens", False) == (t is not None and t > 0)
        assert (e.get("add_vector"), e.get("add_row")) == (("loop.step", t) if t is not None else (None, None))


def test_the_order_of_runs_by_hand():
    c = S.config(10, 8, 1e-5, [S.layer(S.delta(1, 8), None)] * 4, loop=(1, 3, 3))
    assert P.order_of_runs(c) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    for loop in (dict(start=2, stop=2, times=4), None):
        if loop:
            c["loop"] = loop
        else:
            del c["loop"]
        d = describe(c)
        assert [e["layer"] for e in d["spec"]["schedule"]] == [0, 1, 2, 3] and not any("add_vector" in e for e in d["spec"]["schedule"])
        assert "loop.step" not in {t["name"] for t in d["tensor_needs"]}
    assert P.order_of_runs(c) == [(i, None) for i in range(4)]


def test_every_constant_reaches_its_part():
    c = S.CONFIGS["Q1"]
    spec = describe(c)["spec"]
    assert (spec["embedding"], spec["head"], spec["streams"], spec["embedding_scale"], spec["logit_scale"]) == ("embed", "head", 1, 1.0, 1.0)
    assert spec["final_norm"] == dict(kind="rmsnorm", size=64, eps=1e-6, weight="final.norm", one_gain=True)
    L = spec["layers"]
    assert all(b["kind"] == "prenorm" and b["mixer_norm"]["one_gain"] is True for b in L)
    assert L[0]["ff_norm"]["weight"] == "l0.norm2" and L[1]["ff"] is None and L[1]["ff_norm"] is None
    d = L[0]["mixer"]
    assert (d["kind"], d["n_heads"], d["n_kv_heads"], d["head_dim"], d["v_head_dim"], d["taps"], d["eps"], d["key_eps"]) == \
        ("gated_delta", 4, 2, 16, 24, 4, 1e-6, 1e-6)
    assert d["A_log"] == "l0.mix.A_log" and d["v_conv"] == "l0.mix.v.conv" and d["a"] == "l0.mix.a"
    s = L[1]["mixer"]
    assert s["kind"] == "sum" and [m["kind"] for m in s["mixers"]] == ["sigmoid_attention", "time_mixing"]
    a, t = s["mixers"]
    assert (a["n_heads"], a["n_kv_heads"], a["head_dim"], a["v_head_dim"], a["window"], a["taps"], a["softcap"], a["out_scale"]) == \
        (4, 2, 16, 32, 24, 3, 12.0, 0.6)
    assert abs(a["scale"] - 1.7 / 4) < 1e-15 and a["q_bias"] == "l1.mix.left.q.b" and a["o_bias"] == "l1.mix.left.o.b"
    assert a["temp"] == "l1.mix.left.temp" and a["score_bias"] == "l1.mix.left.pb" and a["q_conv"] == "l1.mix.left.q.conv"
    assert a["position"] == dict(kind="rope", head_dim=16, rotary_dim=8, theta=5e4, pairing="half", scaling=None)
    assert (t["n_heads"], t["head_dim"], t["out_scale"], t["mu_w"], t["w2"]) == (3, 20, 1.3, "l1.mix.right.mu.w", "l1.mix.right.w2")
    m = L[2]["mixer"]
    assert (m["kind"], m["n_heads"], m["head_dim"], m["v_head_dim"], m["gate_cap"], m["f_bias"]) == ("matrix_memory", 2, 24, 40, 15.0, "l2.mix.f.b")
    f = L[0]["ff"]
    assert (f["kind"], f["experts"], f["top"], f["score"], f["renormalize"], f["route_scale"], f["weight_on"]) == \
        ("moe", 8, 2, "softmax", False, 2.5, "output")
    assert f["groups"] == dict(count=4, keep=2, top=1) and "correction" not in f and "shared" not in f
    assert f["expert"] == dict(intermediate=24, activation="silu", gate="l0.mlp.e{}.gate", up="l0.mlp.e{}.up", down="l0.mlp.e{}.down")
    # what the configuration leaves out
    q2 = describe(S.CONFIGS["Q2"])["spec"]
    a = q2["layers"][0]["mixer"]["mixers"][0]
    assert a["position"] is None and "window" not in a and a["softcap"] == 0.0 and a["n_kv_heads"] == 3 and a["out_scale"] == 1.0
    assert "q_conv" not in q2["layers"][2]["mixer"] and q2["layers"][1]["ff"]["route_scale"] == 1.0 and "groups" not in q2["layers"][1]["ff"]


def test_faults_are_named():
    from libllm_b200.errors import ConfigError
    base = S.CONFIGS["Q1"]

    def broken(change, match):
        c = copy.deepcopy(base)
        change(c)
        with pytest.raises(ConfigError, match=match):
            describe(c)

    broken(lambda c: c["layers"][0].update(type="conv"), "not known")
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of 'kv_heads'")
    broken(lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple of 'kv_heads'")
    broken(lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "'dims'")
    broken(lambda c: c["layers"][1]["mixer"].pop("right"), "right")
    broken(lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap")
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "'top' exceeds")
    broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "divide")
    broken(lambda c: c["layers"][2]["mlp"]["router"].update(top=3), "fewer experts than 'top'")
    broken(lambda c: c["layers"][0]["mlp"].update(shared=dict(ff=8)), "shared")
    broken(lambda c: c["loop"].update(stop=5), "'start' <= 'stop'")
    broken(lambda c: c.pop("norm"), "norm")


def test_a_run_of_two_mixers_has_one_cache_and_the_state_of_both():
    from libllm_b200.errors import LlmError
    c = S.CONFIGS["Q1"]
    spec = describe(c)["spec"]["layers"][1]["mixer"]
    two = copy.deepcopy(spec)
    two["mixers"] = [two["mixers"][0], two["mixers"][0]]
    from libllm_b200.parts import PartHandle
    with pytest.raises(LlmError, match="one cache"):
        PartHandle("mixer", two)


# ---------------------------------------------------------------- the plain functions by hand
def test_plain_short_convolution():
    u = torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64)
    taps = torch.tensor([[10.0, 1.0]], dtype=torch.float64)                # the last column is the current token's
    assert P.short_conv(u, taps)[:, 0].tolist() == [1.0, 12.0, 23.0]


def test_plain_sigmoid_weights():
    see = P.visible(3, 2)
    assert see.tolist() == [[True, False, False], [True, True, False], [False, True, True]]
    w = P.sigmoid_weights(torch.zeros(3, 3, dtype=torch.float64), see, 2.0, 5.0, 0.0)
    assert w.tolist() == [[0.5, 0.0, 0.0], [0.5, 0.5, 0.0], [0.0, 0.5, 0.5]]      # not normalised over the keys
    s = torch.full((1, 1), 4.0, dtype=torch.float64)
    one = torch.ones(1, 1, dtype=torch.bool)
    assert abs(float(P.sigmoid_weights(s, one, 0.5, 3.0, 0.25)) - 1 / (1 + math.exp(-(3 * math.tanh(2 / 3) + 0.25)))) < 1e-12


def test_plain_recurrences():
    one = lambda *v: torch.tensor(v, dtype=torch.float64).reshape(len(v), 1, 1)
    # delta: S1 = k b v = 0.5; S2 = g S1 + k b (v - k g S1)
    o = P.delta_recurrence(one(1, 1), one(1, 2), one(1, 3), one(0.9, 0.5)[..., 0], one(0.5, 0.25)[..., 0])
    assert torch.allclose(o[:, 0, 0], torch.tensor([0.5, 0.25 + 2 * 0.25 * (3 - 2 * 0.25)], dtype=torch.float64))
    # bonus: the current token's product through u, the state's without it
    o = P.bonus_recurrence(one(1, 1), one(2, 3), one(1, 1), one(0.5, 0.5), torch.tensor([[10.0]], dtype=torch.float64))
    assert o[:, 0, 0].tolist() == [20.0, 2.0 + 30.0]
    # memory: the maximum starts at nought, so a first input gate of -1 beside a forget gate of 0 leaves it there
    o = P.matrix_memory(one(1), one(1), one(4), one(-1)[..., 0], one(0)[..., 0])
    e = math.exp(-1)
    assert abs(float(o) - 4 * e / (max(e, 1.0) + 1e-6)) < 1e-12


def test_plain_choice_among_groups():
    h = torch.eye(4, dtype=torch.float64)[:1]
    w = {"router": torch.zeros(4, 4, dtype=torch.float64)}
    w["router"][:, 0] = torch.tensor([3.0, -5.0, 2.0, 2.5])
    chosen, weight, _ = P.route(h, w, "", dict(experts=4, top=2, scale=2.0, groups=dict(count=2, keep=1)))
    s = torch.softmax(w["router"][:, 0], 0)
    assert chosen.tolist() == [[0, 1]]                                     # the group of the largest expert, its weak neighbour included
    assert torch.allclose(weight[0], 2.0 * s[:2])
