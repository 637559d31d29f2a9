"""Tidenex's configuration, plan, packing of weights and cache needs on the CPU, and the plain implementation against closed forms."""
import copy
import json
import math

import pytest
import torch

import plain_tidenex as plain
import tidenex_models as zoo
from mini_engine_b200.config.model_config import ConfigError, TidenexConfig
from mini_engine_b200.config.registry import get_architecture
from mini_engine_b200.engine.model_runner import plan_cache_groups
from mini_engine_b200.parts import Linear
from mini_engine_b200.weights.loader import WeightsError, expected_disk_tensors, load_weights
from mini_engine_b200.weights.random_init import build_model_from_config_dict


@pytest.mark.parametrize("name", sorted(zoo.ALL))
def test_the_model_asks_for_the_designs_tensors(name):
    cfg, seed, _ = zoo.ALL[name]
    _, model = build_model_from_config_dict(cfg)
    want = {k: tuple(v.shape) for k, v in zoo.tensors(cfg, seed).items()}
    got = {k: tuple(e.shape) for k, e in expected_disk_tensors(model).items() if not e.optional}
    assert got == want
    extra = {k for k, e in expected_disk_tensors(model).items() if e.optional}
    assert extra == {f"l{i}.norm2{b}" for i, layer in enumerate(cfg["layers"]) if layer["mlp"] is None for b in ("", ".b")}


def test_every_number_comes_from_the_file():
    c = TidenexConfig.from_dict(zoo.A)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.loop) == (101, 64, 1e-6, {"start": 1, "stop": 3, "times": 3})
    plan = get_architecture("Tidenex").plan(c)
    (lp, left), (rp, right) = plan.blocks[0].mixer.args["mixers"]
    assert (lp, rp) == ("left.", "right.")
    la, ra = left.args, right.args
    assert (la["num_heads"], la["num_kv_heads"], la["dim"], la["vdim"], la["scale"]) == (4, 2, 16, 24, 0.25)
    assert la["temperature"] == (0.25, 20.0) and la["out_scale"] == 0.7 and la["qk_norm"] == "row" and la["distance_bias"] and la["bias"]
    assert (ra["num_heads"], ra["dim"], ra["vdim"], ra["out_scale"]) == (2, 16, 24, 1.3)
    d = plan.blocks[1].mixer.args
    assert (d["num_heads"], d["num_kv_heads"], d["dim"], d["vdim"], d["diff"]) == (4, 2, 16, 40, 0.45)
    assert plan.shared[d["position_encoding"].key].args == {"rotary_dim": 8, "theta": 500.0}
    assert plan.blocks[1].feed_forward.args["activation"] == "gelu" and plan.blocks[2].feed_forward is None
    assert plan.blocks[4].mixer.args["mixers"][0][1].args["temperature"] is None
    assert plan.tie_word_embeddings and plan.final_norm.args["bias"] == "final.norm.b"
    assert get_architecture("Tidenex").plan(TidenexConfig.from_dict(zoo.B)).blocks[2].mixer.args["position_encoding"] is None
    assert TidenexConfig.from_dict(json.loads(json.dumps(c.to_json_dict()))).layers == c.layers


def test_looped_layers_run_in_passes_with_caches_of_their_own():
    for cfg, want in ((zoo.A, [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]),
                      (zoo.B, [(0, False), (1, False), (0, True), (1, False), (2, False)]),
                      (zoo.C, [(0, False), (1, False), (2, False), (3, False)])):
        plan = get_architecture("Tidenex").plan(TidenexConfig.from_dict(cfg))
        assert [(c.block, c.add_embedding) for c in plan.schedule] == want == plain.layer_runs(cfg)
        assert [c.cache_slot for c in plan.schedule] == list(range(len(want)))
    once = copy.deepcopy(zoo.A)
    once["loop"]["times"] = 1
    assert [r for _, r in TidenexConfig.from_dict(once).layer_runs()] == [False] * 5


def test_cache_rows_and_states():
    _, model = build_model_from_config_dict(zoo.D)
    groups, location, states = plan_cache_groups(model)
    rows = {s: (groups[location[s][0]].num_kv_heads, groups[location[s][0]].head_dim) for s in range(len(model.schedule))}
    # two maps of 40 under a value of 72, a head of 72 four times (looped), two maps of 80 (too wide to be filled), of 16, of 32 / 48
    assert rows == {0: (2, 128), 1: (2, 128), 2: (2, 128), 3: (2, 128), 4: (2, 128), 5: (2, 160), 6: (1, 64), 7: (1, 64)}
    assert {s: states[s][0].shape for s in states} == {1: (2, 32, 56), 2: (2, 32, 56), 3: (2, 32, 56), 4: (2, 32, 56), 7: (1, 8, 16)}


def test_weights_packed_side_by_side_are_loaded_into_their_columns(tmp_path):
    from safetensors.torch import save_file

    class Model(Linear):
        def walk(self):
            return [("m.", self)]
    a, b = torch.randn(6, 3), torch.randn(6, 5)
    save_file({"m.left.o": a, "m.right.o": b}, str(tmp_path / "x.safetensors"))
    part = Model(8, name="o_proj", input_pieces=[("left.o", 3), ("right.o", 5)], out_features=6)
    load_weights(part, str(tmp_path), torch.float32, "cpu")
    assert torch.equal(part.weight, torch.cat((a, b), dim=1))
    x = torch.randn(4, 8)
    assert torch.allclose(x @ part.weight.T, x[:, :3] @ a.T + x[:, 3:] @ b.T, atol=1e-6)
    save_file({"m.left.o": a, "m.right.o": b[:, :4].contiguous()}, str(tmp_path / "x.safetensors"))
    with pytest.raises(WeightsError) as e:
        load_weights(Model(8, name="o_proj", input_pieces=[("left.o", 3), ("right.o", 5)], out_features=6), str(tmp_path), torch.float32, "cpu")
    assert [n for n, _, _ in e.value.wrong_shape] == ["m.right.o"]


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="hgrn2"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(dim=0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "dense"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.pop("vocab"), "vocab"),
])
def test_what_cannot_be_is_refused(edit, text):
    cfg = copy.deepcopy(zoo.A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        TidenexConfig.from_dict(cfg)


# ---- the plain functions against closed forms ---------------------------------------------------------
def test_plain_distance_bias_weighs_equal_scores_by_a_power_of_the_distance():
    """With equal scores the weight of a key at distance d is (1 + r2 d)^-r1, normalised."""
    T, r1, r2 = 9, 1.7, 0.4
    q, k = torch.zeros(T, 1, 4, dtype=torch.float64), torch.zeros(T, 1, 4, dtype=torch.float64)
    v = torch.eye(T, dtype=torch.float64).view(T, 1, T)
    o = plain.causal_attention(q, k, v, 1.0, lambda h, d: r1 * torch.log(1 + r2 * d))
    w = torch.tensor([[(1 + r2 * (i - j)) ** -r1 if j <= i else 0.0 for j in range(T)] for i in range(T)], dtype=torch.float64)
    assert torch.allclose(o[:, 0], w / w.sum(-1, keepdim=True))


def test_plain_temperature_steps():
    p = torch.arange(0, 8, dtype=torch.float64)
    t = plain.temperature(p, 0.5, 4)
    assert torch.allclose(t, torch.tensor([1.0] * 3 + [1 + 0.5 * math.log(2)] * 4 + [1 + 0.5 * math.log(3)], dtype=torch.float64))


def test_plain_recurrence_with_a_constant_gate():
    """A constant gate f and value 1 fill the state to 1 - f^(t+1)."""
    f = torch.full((6, 1, 1), 0.75, dtype=torch.float64)
    o, S = plain.gated_recurrence(torch.ones(6, 1, 1, dtype=torch.float64), f, torch.ones(6, 1, 1, dtype=torch.float64))
    want = torch.tensor([1 - 0.75 ** (t + 1) for t in range(6)], dtype=torch.float64)
    assert torch.allclose(o[:, 0, 0], want) and torch.allclose(S[0, 0, 0], want[-1])
    assert torch.allclose(plain.forget_gate(torch.tensor([-1e3, 0.0, 1e3], dtype=torch.float64), torch.tensor(0.2, dtype=torch.float64)),
                          torch.tensor([0.2, 0.6, 1.0], dtype=torch.float64))


def test_plain_differential_with_equal_maps_and_lambda_is_a_plain_attention():
    """Equal maps give (1 - lambda) a, whose norm leaves the sign and the direction."""
    a = torch.randn(5, 2, 6, dtype=torch.float64)
    out = plain.differential_combine(a, a, 0.3, 0.25, 0.0)
    assert torch.allclose(out, a / a.square().mean(-1, keepdim=True).sqrt() * 0.75)
    w = {"lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.25]), "lq2": torch.tensor([0.0, 1.0]), "lk2": torch.tensor([3.0, 0.1])}
    assert math.isclose(float(plain.differential_lambda(w, "", 0.4)), math.exp(1.0) - math.exp(0.1) + 0.4, rel_tol=1e-6)
