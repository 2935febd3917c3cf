"""Finolix without a GPU: config to parts, tensor names and shapes, layers that run with another layer's tensors, the cache plan, config errors,
the frequencies of the rotated part, and the plain statement's own pieces against hand-made numbers."""

import copy
import math

import pytest
import torch

import finolix_util as FU
from plain import finolix_plain as FP


def _model(cfg):
    from oxr_inference_b200.weights.random_init import shape_only_model

    return shape_only_model(cfg)


def test_architecture_is_found_by_its_single_name():
    from oxr_inference_b200.config.registry import resolve_architecture

    assert resolve_architecture(FU.MODEL_B).name == "Finolix"


def test_tensor_names_and_shapes():
    m = _model(FU.MODEL_A)
    named = {k: tuple(v[2].shape) for k, v in m.named_parameters().items()}
    assert named["embed"] == (127, 52) and named["head"] == (127, 52) and named["final.norm"] == (52,)
    for i in (0, 1, 2, 6):
        assert all(named[f"l{i}.{n}"] == (52,) for n in ("norm1", "norm2", "ls1", "ls2"))
        assert all(named[f"l{i}.hc{q}.in"] == (3,) and named[f"l{i}.hc{q}.out"] == (3,) and named[f"l{i}.hc{q}.mix"] == (3, 3) for q in (1, 2))
    # no feed-forward
    assert {k for k in named if k.startswith("l3.") and ".mix." not in k} == {"l3.norm1", "l3.ls1", "l3.hc1.in", "l3.hc1.out", "l3.hc1.mix"}
    assert named["l0.mix.dq"] == (28, 52) and named["l0.mix.dq.norm"] == (28,) and named["l0.mix.uq"] == (60, 28) and named["l0.mix.sink"] == (3,)
    assert named["l0.mix.dkv"] == (32, 52) and named["l0.mix.dkv.norm"] == (24,) and named["l0.mix.uk"] == (36, 24) and named["l0.mix.uv"] == (60, 24)
    assert named["l0.mix.o"] == (52, 60) and "l0.mix.q" not in named
    assert named["l0.mlp.up"] == (40, 52) and named["l0.mlp.down"] == (52, 40) and "l0.mlp.gate" not in named
    assert named["l1.mix.q"] == (64, 52) and named["l1.mix.k"] == (32, 52) and named["l1.mix.v"] == (48, 52) and named["l1.mix.o"] == (52, 96)
    assert named["l1.mix.q.norm"] == (16,) and named["l1.mix.k.norm"] == (16,) and named["l1.mix.g"] == (4, 52) and "l1.mix.sink" not in named
    assert named["l1.mlp.router"] == (6, 52) and named["l1.mlp.router.b"] == (6,) and named["l1.mlp.e5.gate"] == (24, 52) and "l1.mlp.e6.gate" not in named
    # a layer that runs with another's tensors has none of its own
    assert not [k for k in named if k.startswith(("l4.", "l5."))]


def test_layers_that_run_with_anothers_tensors_have_a_cache_of_their_own():
    m = _model(FU.MODEL_A)
    assert [e.layer for e in m.schedule] == [0, 1, 2, 3, 1, 0, 4] and len(m.blocks) == 5
    e = m.cache_plan.entries
    assert e[4].group == e[1].group and e[4].layer_in_group != e[1].layer_in_group and e[4].store
    assert e[5].group == e[0].group and e[5].layer_in_group != e[0].layer_in_group and e[5].store


def test_weights_of_may_follow_another_weights_of_or_name_a_later_layer():
    from oxr_inference_b200.config.registry import resolve_architecture

    base = FU.latent(mlp=FU.dense())
    cfg = FU.model_config([{**base, "weights_of": 2}, {**base, "weights_of": 0}, base])
    c = resolve_architecture(cfg).config_from_dict(cfg, None)
    assert [layer.owner for layer in c.layers] == [2, 2, 2]
    assert [k for k in _model(cfg).named_parameters() if k.endswith(".ls1")] == ["l2.ls1"]


def test_cache_plan():
    from oxr_inference_b200.parts.base import PagedKVNeed

    plan = _model(FU.MODEL_A).cache_plan
    need = lambda i: plan.groups[plan.entries[i].group].need
    assert need(0) == PagedKVNeed(1, 32, 11, value_dim=0) and need(1) == PagedKVNeed(2, 16, 0, value_dim=24)
    assert need(2) == PagedKVNeed(1, 20, 5, value_dim=0) and need(3) == PagedKVNeed(2, 10, 0) and need(6) == PagedKVNeed(1, 10, 30, value_dim=0)
    assert not plan.states


def test_a_layer_without_a_feed_forward_may_carry_the_tensors_of_one():
    import re

    spec = _model(FU.MODEL_A).spec
    ignored = lambda n: any(re.fullmatch(p, n) for p in spec.ignored_tensors)
    assert all(ignored("l3." + n) for n in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix")) and not ignored("l3.hc1.mix") and not ignored("l3.mlp.up")


def test_blocks_pass_the_streams_on_only_to_blocks_with_as_many():
    from oxr_inference_b200.parts.block import PreNormBlock

    a, b, c = (_model(FU.model_config([FU.latent()], streams=s)).blocks[0] for s in (3, 3, 2))
    assert a.keeps_add_for(b) and not a.keeps_add_for(c) and not a.keeps_add_for(None)
    assert not a.keeps_add_for(PreNormBlock(a.mixer, a.mixer_norm, None, None))


def test_norm_weight_around_zero_becomes_the_factor_in_fp32():
    from oxr_inference_b200.parts.base import NORMS, Runtime

    rt = Runtime(device=torch.device("cpu"), dtype=torch.bfloat16, max_positions=1, status=torch.zeros(4, dtype=torch.int32))
    norm = NORMS.build("rms_norm", rt, size=2, eps=1e-6, around_zero=True)
    norm.assign("weight", torch.tensor([2.0 ** -10, -0.5], dtype=torch.bfloat16))
    assert norm.weight.dtype == torch.float32 and norm.weight.tolist() == [1.0 + 2.0 ** -10, 0.5]


@pytest.mark.parametrize("change,words", [
    (lambda c: c["layers"][0].update(type="mamba2"), "is not one of"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "is not one of"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "lacks 'q_rank'"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rotated part"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=-1), "must be positive"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0}), "lacks 'original'"),
    (lambda c: c["layers"][3]["mixer"].update(heads=3), "not a multiple"),
    (lambda c: c["layers"][3]["mixer"].update(scale="big"), "must be a number"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=0.5), "rot.base"),
    (lambda c: c["layers"][4].update(weights_of=4), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=70), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=0), "does not describe the same layer"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=4), "cannot be chosen"),
    (lambda c: c.pop("streams"), "lacks 'streams'"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(streams=99), "streams"),
    (lambda c: c.pop("norm"), "lacks 'norm'"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_config_errors(change, words):
    from oxr_inference_b200.config.model_config import ConfigError
    from oxr_inference_b200.config.registry import resolve_architecture

    cfg = copy.deepcopy(FU.MODEL_A)
    change(cfg)
    with pytest.raises(ConfigError, match=words):
        resolve_architecture(cfg).config_from_dict(cfg, None)


@pytest.mark.parametrize("dims,base,scaling", [(8, 90.0, FU.ramp()), (16, 1e4, FU.ramp(4.0, 300, 16.0, 1.0)), (2, 50.0, FU.ramp(2.0, 10, 3.0, 2.9)),
                                               (64, 1e5, FU.ramp(40.0, 4096, 32.0, 1.0)), (12, 30.0, None), (6, 3.0, FU.ramp(8.0, 5000, 4.0, 0.01))])
def test_frequencies_and_magnitude_of_the_ramp(dims, base, scaling):
    from oxr_inference_b200.parts.base import POSITION_ENCODINGS, Runtime

    rt = Runtime(device=torch.device("cpu"), dtype=torch.float32, max_positions=1, status=torch.zeros(4, dtype=torch.int32))
    enc = POSITION_ENCODINGS.build("rope_pairs", rt, dims=dims, base=base, scaling={"kind": "ramp", **scaling} if scaling else None)
    freq, magnitude = FP.ramp_frequencies(dims, base, scaling)
    assert enc.freq.tolist() == pytest.approx(freq, rel=1e-14) and enc.magnitude == pytest.approx(magnitude) and not enc.halves


# ------------------------------------------------------------------------------------------------ the plain statement's pieces
def f64(x):
    return torch.tensor(x, dtype=torch.float64)


def test_plain_ramp_by_hand():
    """base e^pi, 4 entries, original 2 pi: the index of t turns is -2 ln t / pi; fast = e^(-pi/2) lies at 1, slow = e^(-3 pi/2) at 3."""
    s = {"factor": 5.0, "original": 2 * math.pi, "fast": math.exp(-math.pi / 2 * 1.01), "slow": math.exp(-3 * math.pi / 2 * 0.99)}
    freq, magnitude = FP.ramp_frequencies(4, math.exp(math.pi), s)
    # lo = floor(1.01) = 1, hi = min(ceil(2.97), 3) = 3: pair 0 keeps its frequency, pair 1 too (ramp 0)
    assert freq == pytest.approx([1.0, math.exp(-math.pi / 2)]) and magnitude == pytest.approx(0.1 * math.log(5.0) + 1.0)
    s["fast"] = math.exp(math.pi / 2)      # index -1: the ramp starts at 0, so pair 1 is a third of the way
    freq, _ = FP.ramp_frequencies(4, math.exp(math.pi), s)
    f = math.exp(-math.pi / 2)
    assert freq == pytest.approx([1.0, f / 5 / 3 + f * 2 / 3])


def test_plain_rotation_pairs_neighbours_or_halves_and_leaves_the_rest():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0] = f64([1.0, 0.0, 0.0, 2.0, 0.0, 7.0])
    pairs, halves = FP.rotate(x, [1.0, 0.1], 3.0, True), FP.rotate(x, [1.0, 0.1], 3.0, False)
    for p in range(3):
        a, b = p * 1.0, p * 0.1
        assert torch.allclose(pairs[p, 0], f64([3 * math.cos(a), 3 * math.sin(a), -6 * math.sin(b), 6 * math.cos(b), 0.0, 7.0]))
        assert torch.allclose(halves[p, 0], f64([3 * math.cos(a), -6 * math.sin(b), 3 * math.sin(a), 6 * math.cos(b), 0.0, 7.0]))


def test_plain_window_counts_the_token_itself_and_the_sink_counts_once():
    seen = FP.visible(5, window=2)
    assert seen[4].tolist() == [False, False, False, True, True] and seen[0].tolist() == [True, False, False, False, False]
    v = f64([[1.0], [10.0]])
    o = FP.attend(f64([[0.0, 9.0], [0.0, math.log(2.0)]]), FP.visible(2), v, f64(math.log(3.0)))
    assert o[:, 0].tolist() == pytest.approx([1 / 4, (1 + 20) / 6])


def test_plain_streams_are_mixed_from_old_to_new():
    x = f64([[[1.0, 2.0]], [[10.0, 20.0]]])                    # two streams, one token
    new = FP.write_streams(x, f64([[0.5, 2.0], [0.0, 1.0]]), f64([3.0, -1.0]), f64([[100.0, 1.0]]))
    assert new.tolist() == [[[0.5 + 300.0, 1.0 + 3.0]], [[2.0 + 10.0 - 100.0, 4.0 + 20.0 - 1.0]]]
    assert FP.read_streams(x, f64([2.0, 0.1])).tolist() == [[3.0, 6.0]]


def test_plain_experts_choose_by_the_biased_logit_and_weigh_by_the_softmax_over_the_chosen():
    h = f64([[2.0]])
    w = {"p.router": f64([[1.0], [0.0], [0.5]]), "p.router.b": f64([0.0, 1.5, -4.0])}
    for e in range(3):
        w.update({f"p.e{e}.gate": f64([[1.0]]), f"p.e{e}.up": f64([[1.0 + e]]), f"p.e{e}.down": f64([[1.0]])})
    unit = 2.0 / (1 + math.exp(-2.0)) * 2.0
    share = math.exp(2.0) / (math.exp(2.0) + math.exp(1.5))
    assert FP.routed_experts(h, w, "p.", {"router": {"experts": 3, "top": 2}}).item() == pytest.approx(share * unit + (1 - share) * 2 * unit)
    assert FP.choice_margin(FP.router_logits(h, w, "p."), 2).item() == pytest.approx(1.5 + 3.0)


def test_plain_forward_looks_at_nothing_ahead():
    cfg = FU.MODEL_A
    torch.manual_seed(0)
    w = {name: torch.randn(info.shape, dtype=torch.float64) * 0.3 for name, (_, _, info) in _model(cfg).named_parameters().items()}
    ids = FU.tokens(cfg, 14, seed=1)
    whole = FP.forward(cfg, w, ids)
    for n in (1, 5, 14):
        assert torch.allclose(FP.forward(cfg, w, ids[:n]), whole[:n], atol=1e-9)
