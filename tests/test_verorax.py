"""Verorax without a GPU: config to parts, tensor names and shapes, layers that run with another layer's tensors, the cache plan (a state row
that holds the mixer's state and the shifted input), config errors, and the plain statement's own pieces against hand-made numbers."""

import copy
import math

import pytest
import torch

import verorax_util as VU
from plain import verorax_plain as VP


def _model(cfg):
    from oxr_inference_b200.weights.random_init import shape_only_model

    return shape_only_model(cfg)


def test_architecture_is_found_by_its_single_name():
    from oxr_inference_b200.config.registry import resolve_architecture

    assert resolve_architecture(VU.MODEL_B).name == "Verorax"


def test_tensor_names_and_shapes():
    m = _model(VU.MODEL_A)
    named = {k: tuple(v[2].shape) for k, v in m.named_parameters().items()}
    assert named["embed"] == (127, 52) and named["head"] == (127, 52) and named["final.norm"] == (52,)
    for i in (0, 1, 2, 6):
        assert all(named[f"l{i}.{n}"] == (52,) for n in ("norm1", "norm1b", "norm2", "norm2b", "shift"))
    assert "l3.norm2" not in named and "l3.norm2b" not in named and named["l3.shift"] == (52,)      # no feed-forward
    assert named["l0.mix.dq"] == (28, 52) and named["l0.mix.dq.norm"] == (28,) and named["l0.mix.uq"] == (60, 28)
    assert named["l0.mix.dkv"] == (32, 52) and named["l0.mix.dkv.norm"] == (24,) and named["l0.mix.uk"] == (36, 24) and named["l0.mix.uv"] == (60, 24)
    assert named["l0.mix.o"] == (52, 60) and "l0.mix.q" not in named and "l0.mix.sink" not in named
    assert named["l0.mlp.gate"] == (56, 52) and named["l0.mlp.down"] == (52, 56)
    assert named["l1.mix.q"] == (80, 52) and named["l1.mix.k"] == (40, 52) and named["l1.mix.v"] == (48, 52) and named["l1.mix.o"] == (52, 96)
    assert named["l1.mix.q.b"] == (80,) and named["l1.mix.k.b"] == (40,) and named["l1.mix.v.b"] == (48,) and "l1.mix.o.b" not in named
    assert all(named[f"l1.mix.{n}"] == (10,) for n in ("lq1", "lk1", "lq2", "lk2"))
    assert named["l1.mlp.router"] == (7, 52) and named["l1.mlp.correction"] == (7,) and named["l1.mlp.e4.gate"] == (24, 52) and "l1.mlp.e5.gate" not in named
    assert named["l2.mix.left.q"] == (64, 52) and named["l2.mix.left.v"] == (48, 52) and named["l2.mix.left.temp"] == (4,) and named["l2.mix.left.g"] == (4, 52)
    assert named["l2.mix.left.q.norm"] == (16,) and named["l2.mix.left.o"] == (52, 96) and "l2.mix.left.out" not in named
    assert named["l2.mix.right.r"] == (36, 52) and named["l2.mix.right.w1"] == (5, 52) and named["l2.mix.right.w2"] == (36, 5) and named["l2.mix.right.w0"] == (36,)
    assert named["l2.mix.right.a"] == (36, 52) and named["l2.mix.right.a.b"] == (36,) and named["l2.mix.right.norm"] == (36,) and named["l2.mix.right.o"] == (52, 36)
    # a layer that runs with another's tensors has none of its own
    assert not [k for k in named if k.startswith(("l4.", "l5."))]


def test_layers_that_run_with_anothers_tensors_have_a_cache_and_a_state_of_their_own():
    m = _model(VU.MODEL_A)
    assert [e.layer for e in m.schedule] == [0, 1, 2, 3, 1, 2, 4] and len(m.blocks) == 5
    e = m.cache_plan.entries
    assert e[4].group == e[1].group and e[4].layer_in_group != e[1].layer_in_group and e[4].store
    assert e[5].group == e[2].group and e[5].layer_in_group != e[2].layer_in_group
    assert len({x.state for x in e}) == 7 and None not in {x.state for x in e}


def test_weights_of_may_follow_another_weights_of_or_name_a_later_layer():
    from oxr_inference_b200.config.registry import resolve_architecture

    base = VU.latent(mlp=VU.dense())
    cfg = VU.model_config([{**base, "weights_of": 2}, {**base, "weights_of": 0}, base])
    c = resolve_architecture(cfg).config_from_dict(cfg, None)
    assert [layer.owner for layer in c.layers] == [2, 2, 2]
    assert [k for k in _model(cfg).named_parameters() if k.endswith(".shift")] == ["l2.shift"]


def test_cache_plan_one_state_row_for_the_mixer_and_the_shifted_input():
    from oxr_inference_b200.parts.base import PagedKVNeed, StateNeed

    plan = _model(VU.MODEL_A).cache_plan
    e = plan.entries
    assert plan.groups[e[0].group].need == PagedKVNeed(1, 24 + 8, 0, value_dim=0) and plan.states[e[0].state] == StateNeed((52,))
    # 32-bit: key rows of both maps side by side beside values of their own size
    assert plan.groups[e[1].group].need == PagedKVNeed(2, 20, 9, value_dim=24) and plan.states[e[1].state] == StateNeed((52,))
    # the recurrence's matrices, then the shifted input
    assert plan.groups[e[2].group].need == PagedKVNeed(2, 16, 11, value_dim=24) and plan.states[e[2].state] == StateNeed((3 * 12 * 12 + 52,))
    odd = _model(VU.model_config([VU.paired(r_heads=1, r_dim=5)], width=39)).cache_plan
    assert odd.states[0] == StateNeed((28 + 40,)), "both parts start at whole 16-byte words"


def test_keys_and_values_of_the_two_maps_stand_at_one_size_in_bfloat16():
    from oxr_inference_b200.parts.base import MIXERS, PagedKVNeed, Runtime

    rt = Runtime(device=torch.device("cpu"), dtype=torch.bfloat16, max_positions=1, status=torch.zeros(4, dtype=torch.int32))
    build = lambda **k: MIXERS.build("differential_attention", rt, None, hidden_size=64, num_heads=4, num_kv_heads=2, scale=1.0, diff=0.5, eps=1e-6, window=5, **k)
    assert build(dim=32, value_dim=64).cache_need() == PagedKVNeed(2, 64, 5) and build(dim=32, value_dim=64).kernel_head_dims() == (64,)
    assert build(dim=10, value_dim=24).cache_need() == PagedKVNeed(2, 32, 5)
    assert build(dim=150, value_dim=64).cache_need() == PagedKVNeed(2, 300, 5, value_dim=64) and build(dim=150, value_dim=64).kernel_head_dims() == ()


def test_the_decay_rank_comes_from_the_checkpoint_shapes():
    from oxr_inference_b200.config.registry import resolve_architecture

    arch = resolve_architecture(VU.MODEL_A)
    cfg = copy.deepcopy(VU.MODEL_A)
    for i in (2, 5):
        cfg["layers"][i]["mixer"]["right"].pop("rank", None)      # the two entries may be one object
    config = arch.config_from_dict(cfg, None)
    rank = lambda shapes: arch.spec_for(config, shapes).layers[2].mixer.params["right"]["params"]["decay_rank"]
    assert rank({"l2.mix.right.w1": (11, 52)}) == 11 and rank(None) == 16


@pytest.mark.parametrize("change,words", [
    (lambda c: c["layers"][0].update(type="retention"), "is not one of"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "is not one of"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "lacks 'q_rank'"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rotated part"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=7), "rot.dims"),
    (lambda c: c["layers"][3]["mixer"].pop("diff"), "lacks 'diff'"),
    (lambda c: c["layers"][3]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][3]["mixer"].update(heads=3), "not a multiple"),
    (lambda c: c["layers"][3]["mixer"].update(scale="big"), "must be a number"),
    (lambda c: c["layers"][2]["mixer"].pop("right"), "lacks 'right'"),
    (lambda c: c["layers"][2]["mixer"].pop("left_scale"), "lacks 'left_scale'"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(base=0.5), "rot.base"),
    (lambda c: c["layers"][4].update(weights_of=4), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=70), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=0), "does not describe the same layer"),
    (lambda c: c["layers"][6]["mlp"]["router"].update(top=8), "cannot be chosen"),
    (lambda c: c["layers"][6]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c.pop("norm"), "lacks 'norm'"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_config_errors(change, words):
    from oxr_inference_b200.config.model_config import ConfigError
    from oxr_inference_b200.config.registry import resolve_architecture

    cfg = copy.deepcopy(VU.MODEL_A)
    change(cfg)
    with pytest.raises(ConfigError, match=words):
        resolve_architecture(cfg).config_from_dict(cfg, None)


# ------------------------------------------------------------------------------------------------ the plain statement's pieces
def f64(x):
    return torch.tensor(x, dtype=torch.float64)


def test_plain_shift_moves_towards_the_previous_token_and_starts_at_zero():
    y = VP.token_shift(f64([[4.0, 1.0], [8.0, 3.0], [0.0, 5.0]]), f64([0.25, 1.0]))
    assert y.tolist() == [[3.0, 0.0], [7.0, 1.0], [2.0, 3.0]]


def test_plain_rotation_pairs_entry_i_with_entry_i_plus_half_and_leaves_the_rest():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 2.0, 7.0
    y = VP.rotate_halves(x, 4, 100.0)
    for p in range(3):
        a, b = p * 1.0, p * 0.1
        want = f64([math.cos(a), -2.0 * math.sin(b), math.sin(a), 2.0 * math.cos(b), 0.0, 7.0])
        assert torch.allclose(y[p, 0], want)


def test_plain_window_counts_the_token_itself():
    seen = VP.visible(5, window=2)
    assert seen[4].tolist() == [False, False, False, True, True] and seen[0].tolist() == [True, False, False, False, False]


def test_plain_delta_rule_takes_out_what_the_old_state_holds_along_the_key():
    """One head of two entries; the second token's key is the first axis: with S_0 known, S_1 = diag(w) S_0 - (a u)(u^T S_0) + k v^T."""
    r, k = f64([[[1.0, 1.0]], [[2.0, 5.0]]]), f64([[[3.0, 4.0]], [[2.0, 0.0]]])
    v, w, a = f64([[[1.0, -1.0]], [[7.0, 0.5]]]), f64([[[0.5, 0.5]], [[0.9, 0.6]]]), f64([[[1.0, 1.0]], [[0.3, 0.8]]])
    o = VP.delta_rule(r, k, v, w, a)
    s0 = torch.outer(k[0, 0], v[0, 0])
    assert torch.allclose(o[0, 0], s0.T @ r[0, 0])
    s1 = torch.stack([0.9 * s0[0] - 0.3 * s0[0] + 2.0 * v[1, 0], 0.6 * s0[1]])
    assert torch.allclose(o[1, 0], s1.T @ r[1, 0], rtol=1e-6)      # the unit key's length has 1e-6 under its root


def test_plain_map_weight():
    w = {"lq1": f64([1.0, 2.0]), "lk1": f64([0.5, 0.25]), "lq2": f64([0.0, 1.0]), "lk2": f64([3.0, 0.5])}
    assert VP.map_weight(w, "", 0.3).item() == pytest.approx(math.exp(1.0) - math.exp(0.5) + 0.3)


def test_plain_experts_choose_by_the_corrected_score_and_weigh_by_the_score():
    """Two experts and one identity expert, top 1: the correction turns the choice over, the weight stays the softmax score."""
    h = f64([[2.0]])
    w = {"p.router": f64([[1.0], [0.0], [0.5]]), "p.correction": f64([0.0, 0.0, 5.0])}
    for e in range(2):
        w.update({f"p.e{e}.gate": f64([[1.0]]), f"p.e{e}.up": f64([[1.0 + e]]), f"p.e{e}.down": f64([[1.0]])})
    s = torch.softmax(f64([2.0, 0.0, 1.0]), 0)
    mlp = {"router": {"experts": 2, "identity": 1, "top": 1}}
    assert VP.routed_experts(h, w, "p.", mlp).item() == pytest.approx((s[2] * 2.0).item())
    w["p.correction"] = f64([0.0, 0.9, -1.0])
    unit = 2.0 / (1 + math.exp(-2.0)) * 4.0
    assert VP.routed_experts(h, w, "p.", mlp).item() == pytest.approx((s[1] * unit).item())
    assert VP.choice_margin(VP.router_scores(h, w, "p."), w["p.correction"], 1).item() == pytest.approx((s[1] + 0.9 - s[0]).item())


def test_plain_forward_looks_at_nothing_ahead():
    cfg = VU.MODEL_A
    torch.manual_seed(0)
    w = {name: torch.randn(info.shape, dtype=torch.float64) * 0.3 for name, (_, _, info) in _model(cfg).named_parameters().items()}
    ids = VU.tokens(cfg, 14, seed=1)
    whole = VP.forward(cfg, w, ids)
    for n in (1, 5, 14):
        assert torch.allclose(VP.forward(cfg, w, ids[:n]), whole[:n], atol=1e-9)
