"""Kuterax's configuration, plan and cache needs on the CPU, and the plain implementation against closed forms."""
import copy
import json
import math

import pytest
import torch

import kuterax_models as zoo
import plain_kuterax as plain
from mini_engine_b200.config.model_config import ConfigError, KuteraxConfig
from mini_engine_b200.config.registry import get_architecture
from mini_engine_b200.engine.model_runner import plan_cache_groups
from mini_engine_b200.parts import FrequencyRotary
from mini_engine_b200.weights.loader import expected_disk_tensors
from mini_engine_b200.weights.random_init import build_model_from_config_dict


@pytest.mark.parametrize("name", sorted(zoo.ALL))
def test_the_model_asks_for_the_designs_tensors(name):
    cfg, seed, _ = zoo.ALL[name]
    _, model = build_model_from_config_dict(cfg)
    want = {k: tuple(v.shape) for k, v in zoo.tensors(cfg, seed).items()}
    assert {k: tuple(e.shape) for k, e in expected_disk_tensors(model).items() if not e.optional} == want
    assert {k for k, e in expected_disk_tensors(model).items() if e.optional} == {f"l{i}.ls2" for i, l in enumerate(cfg["layers"]) if l["mlp"] is None}


def test_every_number_comes_from_the_file():
    c = KuteraxConfig.from_dict(zoo.A)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.max_position_embeddings, c.loop) == (101, 64, 1e-6, 512, {"start": 1, "stop": 3, "times": 3})
    plan = get_architecture("Kuterax").plan(c)
    assert plan.position_table == ("pos", 512) and plan.pass_vectors == ("loop.step", 3) and plan.pass_input == "loop.in"
    r = plan.blocks[0].mixer.args
    assert (r["num_heads"], r["dim"], r["vdim"], r["decay"]) == (2, 16, 24, [0.9, 0.99])
    (lp, left), (rp, right) = plan.blocks[1].mixer.args["mixers"]
    la, ra = left.args, right.args
    assert (lp, rp, la["num_heads"], la["num_kv_heads"], la["dim"], la["vdim"], la["scale"]) == ("left.", "right.", 4, 2, 16, 24, 0.25)
    assert la["mask"] == ("window", 20) and la["sink"] == "one" and la["head_gate"] and la["bias"] and not la["output_bias"] and la["qk_norm"] == "before"
    assert plan.shared[la["position_encoding"].key].args == {"rotary_dim": 8, "theta": 500.0,
                                                             "scaling": {"factor": 8.0, "original": 256.0, "fast": 16.0, "slow": 1.0}}
    assert (ra["num_heads"], ra["vdim"], ra["state"], ra["groups"], ra["taps"], ra["norm_groups"]) == (4, 8, 16, 2, 4, 2)
    f = plan.blocks[1].feed_forward.args
    assert (f["num_experts"], f["top"], f["expert_size"], f["groups"], f["weight_scale"], f["routing"]) == (8, 3, 32, (4, 2), 0.7, "softmax_groups")
    assert f["shared"] == {"intermediate_size": 24, "activation": "relu_squared"} and f["activation"] == "relu_squared"
    assert plan.blocks[2].feed_forward is None and not plan.tie_word_embeddings
    d = get_architecture("Kuterax").plan(KuteraxConfig.from_dict(zoo.D))
    assert "shared" not in d.blocks[3].feed_forward.args and d.pass_vectors == ("loop.step", 4)
    assert get_architecture("Kuterax").plan(KuteraxConfig.from_dict(zoo.C)).pass_input is None
    assert KuteraxConfig.from_dict(json.loads(json.dumps(c.to_json_dict()))).layers == c.layers


def test_looped_layers_run_in_passes_with_caches_of_their_own():
    for cfg, want in ((zoo.A, [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]),
                      (zoo.B, [(0, 0), (1, None), (0, 1), (1, None), (2, None)]), (zoo.C, [(0, None), (1, None), (2, None)])):
        plan = get_architecture("Kuterax").plan(KuteraxConfig.from_dict(cfg))
        assert [(c.block, c.add_row) for c in plan.schedule] == want == plain.layer_runs(cfg)
        assert [c.join_embedding for c in plan.schedule] == [t is not None for _, t in want]
        assert [c.cache_slot for c in plan.schedule] == list(range(len(want)))


def test_cache_rows_and_states():
    _, model = build_model_from_config_dict(zoo.D)
    groups, location, states = plan_cache_groups(model)
    rows = {s: (groups[location[s][0]].num_kv_heads, groups[location[s][0]].head_dim, groups[location[s][0]].window) for s in location}
    assert rows == {0: (2, 128, 7), 1: (2, 128, 64), 2: (2, 128, 64), 3: (2, 128, 64), 4: (2, 128, 64), 5: (2, 144, 1)}
    shapes = {s: {n.name: n.shape for n in states[s]} for s in states}
    assert shapes[0] == {"S": (4, 24, 16)}                                                   # one tap: no inputs to keep
    assert shapes[1] == shapes[4] == {"S": (6, 20, 12), "conv": (5, 72 + 2 * 3 * 20)}
    assert shapes[5] == {"S": (1, 32, 32), "conv": (3, 96)} and shapes[6] == {"S": (1, 72, 8)}


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="gla"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.0]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "moe"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "choices"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "choices"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.pop("max_positions"), "max_positions"),
])
def test_what_cannot_be_is_refused(edit, text):
    cfg = copy.deepcopy(zoo.A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        KuteraxConfig.from_dict(cfg)


# ---- frequencies, and the plain functions against closed forms ---------------------------------------------
@pytest.mark.parametrize("dims, base, scaling", [(64, 1e4, (4.0, 4096, 32.0, 1.0)), (24, 1e4, (8.0, 256, 16.0, 1.0)), (8, 500.0, (3.0, 100, 6.0, 0.5)),
                                                 (2, 50.0, (2.0, 64, 4.0, 1.0)), (96, 1e6, (16.0, 64, 40.0, 9.0)), (20, 2000.0, (1.0, 300, 8.0, 2.0))])
def test_yarn_frequencies_of_the_rotation_part(dims, base, scaling):
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling))
    rope = FrequencyRotary(dims, base, sc)
    want, magnitude = plain.yarn_frequencies(dims, base, sc)
    assert torch.allclose(torch.tensor(rope.frequencies(), dtype=torch.float64), torch.tensor(want, dtype=torch.float64), rtol=1e-12)
    assert math.isclose(rope.magnitude, magnitude) and math.isclose(magnitude, 1.0 + 0.1 * math.log(scaling[0]))
    assert FrequencyRotary(dims, base).magnitude == 1.0


def test_plain_yarn_keeps_fast_frequencies_and_divides_slow_ones():
    f, _ = plain.yarn_frequencies(64, 1e4, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    plain_f, _ = plain.yarn_frequencies(64, 1e4)
    ratio = [b / a for a, b in zip(f, plain_f)]
    assert math.isclose(ratio[0], 1.0) and math.isclose(ratio[-1], 4.0) and all(b >= a - 1e-12 for a, b in zip(ratio, ratio[1:]))
    for i, r in enumerate(ratio):                      # the wavelength fits more than fast times / fewer than slow times into original
        turns = 4096 * plain_f[i] / (2 * math.pi)
        assert (r == pytest.approx(1.0)) if turns > 40 else True
        assert (r == pytest.approx(4.0)) if turns < 0.7 else True


def test_plain_window_and_the_one_in_the_denominator():
    """Equal scores of zero: every seen key weighs 1 / (n + 1)."""
    T, w = 7, 3
    q = torch.zeros(T, 1, 2, dtype=torch.float64)
    v = torch.eye(T, dtype=torch.float64).view(T, 1, T)
    o = plain.window_attention(q, q, v, 1.0, w)[:, 0]
    for i in range(T):
        n = min(i + 1, w)
        assert torch.allclose(o[i], torch.tensor([1 / (n + 1) if i - w < j <= i else 0.0 for j in range(T)], dtype=torch.float64))


def test_plain_state_space_scan_with_constant_inputs():
    """Constant dt, B = C = x = 1: S_t = dt (1 - a^(t+1)) / (1 - a) with a = exp(-exp(A_log) dt); y adds D."""
    T, dt, A_log, D = 6, 0.3, 0.2, 0.5
    one = torch.ones(T, 1, 1, dtype=torch.float64)
    f = lambda x: torch.tensor([x], dtype=torch.float64)
    y, S = plain.state_space_scan(one, one, one, torch.full((T, 1), dt, dtype=torch.float64), f(A_log), f(D))
    a = math.exp(-math.exp(A_log) * dt)
    want = torch.tensor([dt * (1 - a ** (t + 1)) / (1 - a) for t in range(T)], dtype=torch.float64)
    assert torch.allclose(y[:, 0, 0], want + D) and torch.allclose(S[0, 0, 0], want[-1])
    assert torch.allclose(plain.softplus(f(-800.0)), f(0.0)) and torch.allclose(plain.softplus(f(0.0)), f(math.log(2))) and plain.softplus(f(90.0)) == 90.0


def test_plain_retention_and_convolution():
    one = torch.ones(5, 1, 1, dtype=torch.float64)
    o, _ = plain.retention_scan(one, one, one, [0.5])
    assert torch.allclose(o[:, 0, 0], torch.tensor([2 - 0.5 ** t for t in range(5)], dtype=torch.float64))
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    c = plain.causal_conv(u, torch.tensor([[10.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert torch.allclose(c[:, 0], torch.tensor([1.5, 12.5, 24.5], dtype=torch.float64))


def test_plain_routing_chooses_inside_the_best_groups_by_the_largest_score():
    """The group with the largest single score wins although the other one has the larger sum and the second largest score."""
    z = torch.tensor([2.0, -9.0, -9.0, 1.9, 1.8, 1.7], dtype=torch.float64)
    chosen, w = plain.route(z, 2, 2, 1, 3.0)
    s = torch.softmax(z, -1)
    assert chosen == [0, 1] and torch.allclose(torch.stack(w), 3.0 * s[[0, 1]])
    assert plain.route(z, 2, 2, 2, 1.0)[0] == [0, 3]
