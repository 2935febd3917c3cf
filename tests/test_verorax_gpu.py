"""Verorax on the GPU against the plain statement in ``tests/plain/verorax_plain.py``: each mechanism alone, the stream after every layer,
whole prompts against token-by-token decoding, portions down to two tokens, batches of unequal requests, pages and slots that are used
again, marked keys far back, at page borders and just inside and outside a window, long decoding, greedy generation through the engine, and
the new kernels against their formulas."""

import math

import pytest
import torch

import verorax_util as VU
from plain import verorax_plain as VP
from util import Replay

pytestmark = pytest.mark.gpu

DEV = "cuda"

CLOSE_CALL = 0.008
"""bfloat16 rows at which some router of the plain model decided by less than this (a difference of softmax scores) are not compared:
a score that differs by a rounding step may choose another expert there, for no fault. (32-bit compares every row.)"""


def close(got, want, dtype, what, margins=None, spreading=False):
    """32-bit: every row within 2e-4 of the row's spread. bfloat16: within 8e-2, one row in twenty (at least one) up to 0.25. ``spreading``: the
    model has routers below attention layers, so a choice that a bfloat16 rounding step turns over at one token reaches later tokens, and no
    row can be cleared by its own margins alone: then nine clear rows in ten within 8e-2 and the median within 4e-2 (32-bit still compares
    every row)."""
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    d = (got - want) - (got - want).mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.std(-1).clamp_min(1e-6)
    if dtype == "float32":
        assert err.max() <= 2e-4, f"{what}: row {int(err.argmax())} is off by {err.max():.2e} of the row's spread (limit 2e-04)"
        return
    if margins is not None:
        clear = margins >= CLOSE_CALL
        assert clear.float().mean() >= 0.4 or len(clear) < 12, f"{what}: most rows are close calls of a router; the test compares too little"
        err = torch.where(clear, err, torch.zeros_like(err))
    over = int((err > 8e-2).sum())
    if spreading:
        assert over <= max(1, len(err) // 10) and err.median() <= 4e-2, (
            f"{what}: {over} of {len(err)} rows are off by more than 8e-02 of the row's spread, the median by {err.median():.2e}")
        return
    assert err.max() <= 0.25 and over <= max(1, len(err) // 20), (
        f"{what}: {over} of {len(err)} rows are off by more than 8e-02 of the row's spread, row {int(err.argmax())} by {err.max():.2e}")


def runner_for(folder, dtype, *, page_size=8, num_pages=64, max_requests=4):
    from oxr_inference_b200.engine.runtime import ModelRunner

    return ModelRunner.from_folder(folder, dtype=dtype, page_size=page_size, num_pages=num_pages, max_requests=max_requests)


def feed(runner, rc, ids, lo, hi, want=None):
    from oxr_inference_b200.engine.batch import StepEntry

    assert runner.cache.reserve(rc, hi)
    return StepEntry(rc, ids[lo:hi], list(range(hi - lo)) if want is None else want)


def run_cut(runner, ids, cuts):
    """One request alone, cut into portions; logits of every position."""
    rc = runner.cache.open("r")
    rows, at = [], 0
    for c in cuts:
        rows.append(runner.step([feed(runner, rc, ids, at, at + c)]))
        at += c
    assert at == len(ids)
    runner.check()
    runner.cache.close(rc)
    runner.cache.check()
    return torch.cat(rows)


# ------------------------------------------------------------------------------------------------ each mechanism alone
L, D, P, MOE, DENSE, CFG = VU.latent, VU.differential, VU.paired, VU.moe, VU.dense, VU.model_config
SINGLE = {
    "latent_alone": CFG([L()]),
    "latent_one_head_two_rotated_entries": CFG([L(heads=1, rot_dim=2, dim=4, kv_rank=16, q_rank=8)]),
    "latent_tiled_sizes": CFG([L(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=32)], width=64),
    "latent_odd_sizes": CFG([L(heads=3, dim=7, rot_dim=6, vdim=9, kv_rank=13, q_rank=11)], width=39),
    "latent_wide_row": CFG([L(heads=2, dim=32, rot_dim=32, vdim=16, kv_rank=256, q_rank=48, scale=0.2)]),
    "differential_alone": CFG([D()]),
    "differential_values_as_wide_as_both_maps": CFG([D(heads=6, kv_heads=2, dim=16, vdim=32, size=13)], width=64),
    "differential_values_wider_than_both_maps": CFG([D(heads=2, kv_heads=1, dim=8, vdim=64, size=40)]),
    "differential_values_smaller_than_a_map": CFG([D(heads=4, kv_heads=4, dim=40, vdim=16, size=6, scale=0.2)]),
    "differential_window_of_one": CFG([D(size=1)]),
    "differential_window_beyond_the_prompt": CFG([D(size=500)]),
    "differential_odd_sizes": CFG([D(heads=3, kv_heads=1, dim=7, vdim=11, size=5, diff=0.8)], width=39),
    "differential_tma_sizes": CFG([D(heads=6, kv_heads=3, dim=32, vdim=64, size=21, scale=0.3)], width=64),
    "pair_alone": CFG([P()]),
    "pair_equal_sizes_all_rotated": CFG([P(heads=6, kv_heads=3, dim=32, vdim=32, rot=32, size=17, scale=0.2, r_heads=2, r_dim=16)], width=64),
    "pair_two_rotated_entries": CFG([P(rot=2, base=5.0, size=3)]),
    "pair_left_only": CFG([P(right_scale=0.0)]),
    "pair_right_only": CFG([P(left_scale=0.0, right_scale=1.0)]),
    "pair_one_wide_recurrent_head": CFG([P(left_scale=0.1, right_scale=1.0, r_heads=1, r_dim=130, rank=2)]),
    "pair_tma_sizes": CFG([P(heads=2, kv_heads=1, dim=64, vdim=64, rot=16, size=30, scale=0.15, r_heads=1, r_dim=64)], width=64),
    "dense_feed_forward": CFG([D(mlp=DENSE())]),
    "dense_feed_forward_wide": CFG([D(mlp=DENSE(ff=96))], width=64),
    "experts": CFG([D(mlp=MOE())]),
    "experts_without_identity": CFG([D(mlp=MOE(identity=0, top=2))]),
    "experts_mostly_identity": CFG([D(mlp=MOE(experts=1, identity=6, top=4))]),
    "experts_top_one": CFG([D(mlp=MOE(experts=6, identity=3, top=1))]),
    "experts_all_chosen": CFG([D(mlp=MOE(experts=3, identity=2, top=5, ff=20))]),
    "experts_odd_sizes": CFG([D(mlp=MOE(experts=7, identity=1, top=3, ff=9))], width=39),
    "one_layer_three_times": CFG([P(mlp=DENSE(ff=24)), VU.again([P(mlp=DENSE(ff=24))], 0), VU.again([P(mlp=DENSE(ff=24))], 0)]),
    "weights_of_a_later_layer": CFG([{**L(), "weights_of": 1}, L()]),
    "no_feed_forward_between_layers_that_have_one": CFG([L(mlp=DENSE()), D(), P(), L(mlp=DENSE(ff=24))]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_mechanism(name, dtype, tmp_path):
    cfg = SINGLE[name]
    folder = VU.make_folder(tmp_path, cfg, name, seed=5)
    ids = VU.tokens(cfg, 61, seed=1)
    want = VU.plain_logits(folder, ids)
    r = runner_for(folder, dtype)
    mg = VU.router_margins(folder, ids)
    close(run_cut(r, ids, [61]), want, dtype, f"{name}, whole prompt", mg)
    close(run_cut(r, ids, [29] + [1] * 32), want, dtype, f"{name}, 29 tokens then one by one", mg)
    close(run_cut(r, ids, [2, 3, 2, 11, 2, 17, 1, 2, 21]), want, dtype, f"{name}, portions", mg)


@pytest.mark.parametrize("width,ff,experts,identity,top", [(64, 16, 6, 2, 2), (40, 20, 5, 1, 3), (72, 36, 3, 5, 2), (39, 9, 4, 0, 3)])
def test_experts_grouped_by_expert_equal_the_two_products_form(width, ff, experts, identity, top, tmp_path):
    """From ``grouped_min_rows`` tokens on every expert multiplies only the rows that chose it; below, all experts are two products. The identity
    experts' share joins in the last kernel or as a pass of its own. Both against the plain sum, in both dtypes, also for odd widths."""
    cfg = CFG([D(mlp=MOE(experts=experts, identity=identity, top=top, ff=ff))], width=width)
    folder = VU.make_folder(tmp_path, cfg, "grouped", seed=8)
    ids = VU.tokens(cfg, 70, seed=3)
    want, mg = VU.plain_logits(folder, ids), VU.router_margins(folder, ids)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(folder, dtype)
        part = r.model.blocks[0].feed_forward
        for rows in (0, 8):
            part.grouped_min_rows = rows
            close(run_cut(r, ids, [40, 5, 25]), want, dtype, f"experts, grouped from {rows} rows on, {dtype}", mg)


def test_layer_results_one_by_one(tmp_path):
    """The stream after every layer against the plain statement's, in 32-bit (no block leaves its last add to the next one here)."""
    from oxr_inference_b200.engine.batch import StepEntry

    for name, cfg in (("A", VU.MODEL_A), ("B", VU.MODEL_B)):
        folder = VU.make_folder(tmp_path, cfg, name, seed=2)
        ids = VU.tokens(cfg, 23, seed=6)
        plain_cfg, w = VP.read_model(folder, torch.float64)
        want: list = []
        VP.forward(plain_cfg, w, ids, streams=want)
        r = runner_for(folder, "float32")
        got = []
        for b in r.model.blocks:
            def wrapped(*a, _f=b.forward, **k):
                out = _f(*a, **k)
                assert out[0] is None
                got.append(out[1].clone())
                return out
            b.forward, b.keeps_add_for = wrapped, lambda after: False
        rc = r.cache.open("r")
        assert r.cache.reserve(rc, len(ids))
        r.step([StepEntry(rc, ids, [len(ids) - 1])])
        r.cache.close(rc)
        assert len(got) == len(want) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(got, want)):
            err = (a.double().cpu() - b).abs().max() / b.abs().max()
            assert err < 2e-5, f"model {name}, layer {i} ({cfg['layers'][i]['type']}): off by {err:.2e} of the stream's largest entry"


# ------------------------------------------------------------------------------------------------ whole models, every cutting
MODELS = {"A": VU.MODEL_A, "B": VU.MODEL_B, "C": VU.MODEL_C}
SPREADING = {"A": True, "B": True, "C": False}
"""Whether a model has routers below attention layers (see ``close``)."""


@pytest.fixture(scope="module", params=[(m, d) for m in sorted(MODELS) for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def model(request, tmp_path_factory):
    name, dtype = request.param
    # 32-bit runs take the weights at full strength and compare every row at 2e-4; 16-bit runs of these deep models take them milder
    folder = VU.make_folder(tmp_path_factory.mktemp(f"verorax_{name}_{dtype}"), MODELS[name], name, seed=11, strength=1.0 if dtype == "float32" else 0.25)
    return name, dtype, folder, runner_for(folder, dtype, page_size=8, num_pages=40)


def test_whole_prompt_equals_token_by_token(model):
    name, dtype, folder, r = model
    cfg = MODELS[name]
    for n in (1, 2, 9, 75):
        ids = VU.tokens(cfg, n, seed=2)
        want, mg = VU.plain_logits(folder, ids), VU.router_margins(folder, ids)
        close(run_cut(r, ids, [n]), want, dtype, f"{name}: whole prompt of {n}", mg, SPREADING[name])
        close(run_cut(r, ids, [1] * n), want, dtype, f"{name}: {n} tokens one by one", mg, SPREADING[name])


def test_portions_of_several_sizes(model):
    name, dtype, folder, r = model
    ids = VU.tokens(MODELS[name], 120, seed=3)
    want, mg = VU.plain_logits(folder, ids), VU.router_margins(folder, ids)
    for cuts in ([2] * 60, [7, 2, 13, 3, 2, 31, 1, 16, 2, 17, 8, 18], [33, 33, 33, 21], [119, 1], [15, 16, 17, 32, 40]):
        close(run_cut(r, ids, cuts), want, dtype, f"{name}: portions {cuts[:4]}...", mg, SPREADING[name])


def test_long_decoding(model):
    name, dtype, folder, r = model
    ids = VU.tokens(MODELS[name], 260, seed=4)
    close(run_cut(r, ids, [4] + [1] * 256), VU.plain_logits(folder, ids), dtype, f"{name}: 256 decoded tokens", VU.router_margins(folder, ids), SPREADING[name])


def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(model):
    """Four live requests at most, 40 pages of 8 tokens: the lengths below need far more over time, so pages and state slots come back and are
    handed out again (a slot's shifted input and recurrence matrices must start at zero); every request's logits equal those it gets alone."""
    name, dtype, folder, r = model
    cfg = MODELS[name]
    lengths = [97, 3, 64, 30, 1, 121, 45, 18, 70]
    todo = [(f"q{i}", VU.tokens(cfg, n, seed=20 + i)) for i, n in enumerate(lengths)]
    live, got, cuts = {}, {}, {}
    step = 0
    while todo or live:
        while todo and len(live) < 4:
            key, ids = todo.pop(0)
            rc = r.cache.open(key)
            assert rc is not None
            live[key] = [rc, ids, 0]
        entries, order = [], []
        for k, (key, (rc, ids, at)) in enumerate(sorted(live.items())):
            if (step + k) % 3 == 0 and at > 0 and len(live) > 1:
                continue                                   # a request may sit a step out
            left = len(ids) - at
            c = 1 if at >= len(ids) // 2 else min(left, [2, 5, 16, 3, 29][(step + k) % 5])   # portions first, then single tokens
            if r.cache.free_pages * 8 < c + 8:
                continue
            entries.append(feed(r, rc, ids, at, at + c))
            order.append((key, c))
        if not entries:   # everything sat out or lacked pages: let the longest go on alone
            key, (rc, ids, at) = max(live.items(), key=lambda kv: kv[1][2])
            entries, order = [feed(r, rc, ids, at, at + 1)], [(key, 1)]
        out = r.step(entries)
        row = 0
        for key, c in order:
            got.setdefault(key, []).append(out[row:row + c])
            cuts.setdefault(key, []).append(c)
            row += c
            live[key][2] += c
            if live[key][2] == len(live[key][1]):
                r.cache.close(live.pop(key)[0])
        step += 1
    r.check()
    r.cache.check()
    assert sum(-(-n // 8) for n in lengths) > 40, "the requests never needed a page twice"
    for i, n in enumerate(lengths):
        ids = VU.tokens(cfg, n, seed=20 + i)
        mixed = torch.cat(got[f"q{i}"])
        if dtype == "bfloat16" and SPREADING[name]:
            # what the mix must not change is told apart from what 16 bits do to a deep model with routers: the same request alone, cut alike
            alone = run_cut(r, ids, cuts[f"q{i}"]).float().cpu()
            d = (mixed.float().cpu() - alone) - (mixed.float().cpu() - alone).mean(-1, keepdim=True)
            err = d.pow(2).mean(-1).sqrt() / alone.std(-1).clamp_min(1e-6)
            assert int((err > 3e-2).sum()) <= n // 20, f"{name}: request {i} of {n} tokens differs in the mix from itself alone: row {int(err.argmax())} by {err.max():.2e}"
        else:
            close(mixed, VU.plain_logits(folder, ids), dtype, f"{name}: request {i} of {n} tokens in the mix", VU.router_margins(folder, ids))


def test_far_keys_and_a_long_lived_state(tmp_path):
    """A prompt of 700 tokens with peaked attention and slowly decaying state: the last logits rest on keys from hundreds of tokens back,
    across dozens of pages, and on what the recurrence has carried; in 32-bit a lost key shows."""
    cfg = CFG([L(heads=4, dim=16, rot_dim=16, vdim=32, kv_rank=48, q_rank=32, base=1e4, scale=0.5, mlp=DENSE(ff=40)),
               P(heads=2, kv_heads=1, dim=64, vdim=64, rot=32, base=1e4, size=300, scale=0.2, r_heads=2, r_dim=32, rank=4),
               D(heads=4, kv_heads=2, dim=16, vdim=32, size=150, scale=0.5, mlp=MOE(ff=16, experts=4, identity=2, top=2))], width=64, vocab=180)
    ids = VU.tokens(cfg, 700, seed=9)
    for dtype in ("float32", "bfloat16"):        # the model's router stands in its last layer; 16-bit runs take the weights milder, as above
        folder = VU.make_folder(tmp_path, cfg, f"far_{dtype}", seed=3, sharpen=4.0, strength=1.0 if dtype == "float32" else 0.25)
        want, mg = VU.plain_logits(folder, ids), VU.router_margins(folder, ids)
        r = runner_for(folder, dtype, page_size=16, num_pages=50)
        close(run_cut(r, ids, [650] + [1] * 50), want, dtype, f"{dtype}: 650 tokens, then 50 one by one", mg)
        close(run_cut(r, ids, [255, 257, 2, 186]), want, dtype, f"{dtype}: portions that end beside page borders", mg)


def test_windows_release_their_pages_and_nothing_else(tmp_path):
    cfg = CFG([D(size=9), P(size=20), L()])
    r = runner_for(VU.make_folder(tmp_path, cfg, "windows", seed=1), "float32", page_size=4, num_pages=40)
    rc = r.cache.open("r")
    ids = VU.tokens(cfg, 60, seed=1)
    r.step([feed(r, rc, ids, 0, 60)])
    by_window = {g.need.window: sum(p >= 0 for p in rc.tables[i]) for i, g in enumerate(r.cache.plan.groups)}
    assert by_window == {9: 2, 20: 5, 0: 15}      # the next query sits at 60 and sees keys from 52, from 41 and from 0 on
    r.cache.close(rc)
    r.cache.check()


def test_replay_program_runs_the_design(tmp_path):
    cfg = VU.MODEL_A
    folder = VU.make_folder(tmp_path, cfg, "A", seed=11)
    ids_a, ids_b = VU.tokens(cfg, 50, seed=7), VU.tokens(cfg, 9, seed=8)
    r = Replay(folder, "float32", tmp_path / "out", max_tokens=128, page_size=16)
    got = r.step([{"id": "a", "tokens": ids_a[:31], "want": [0, 30]}, {"id": "b", "tokens": ids_b[:2], "want": []}])
    close(got, VU.plain_logits(folder, ids_a)[[0, 30]], "float32", "replay: first step")
    assert r.step([{"id": "b", "tokens": ids_b[2:8], "want": []}]) is None
    got = r.step([{"id": "a", "tokens": ids_a[31:], "want": [18]}, {"id": "b", "tokens": ids_b[8:], "want": [0]}], end=["a", "b"])
    close(got, torch.stack([VU.plain_logits(folder, ids_a)[49], VU.plain_logits(folder, ids_b)[8]]), "float32", "replay: last step")
    assert r.close() == 0


# ------------------------------------------------------------------------------------------------ greedy generation through the engine
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_engine(which, graphs, tmp_path):
    from oxr_inference_b200.config import EngineSettings
    from oxr_inference_b200.engine.api import Engine, SamplingParams

    cfg = MODELS[which]
    folder = VU.make_folder(tmp_path, cfg, which, seed=11)
    plain_cfg, w = VP.read_model(folder, torch.float64)
    prompts = [VU.tokens(cfg, n, seed=30 + n) for n in (5, 23, 1, 40, 12, 9)]
    engine = Engine(folder, EngineSettings(dtype="float32", num_pages=48, page_size=8, max_running=3, max_step_tokens=32, prefill_chunk=16,
                                           cuda_graphs=graphs))
    done = engine.generate(prompts, SamplingParams(max_tokens=14, ignore_eos=True))
    compared = 0
    for prompt, c in zip(prompts, done):
        want, gaps = VP.greedy(plain_cfg, w, prompt, 14)
        for a, b, gap in zip(c.token_ids, want, gaps):
            if gap < 1e-3:
                break          # a near-tie: from here on the two may differ for no fault
            assert a == b, f"prompt of {len(prompt)}: generated {c.token_ids}, the plain implementation {want}"
            compared += 1
    assert compared >= 60
    if graphs:
        assert engine.counters["graph_steps"] > 0


def test_command_line_generates_with_the_design(tmp_path):
    import json
    import subprocess
    import sys

    import util

    cfg = VU.MODEL_A
    folder = VU.make_folder(tmp_path, cfg, "A", seed=14)
    plain_cfg, w = VP.read_model(folder, torch.float64)
    cmd = [sys.executable, "-m", "oxr_inference_b200", "--model", str(folder), "--prompt-ids", "5,17,3", "--prompt-ids", "9 8 7 6 11 2",
           "--max-tokens", "6", "--dtype", "float32", "--num-pages", "32", "--max-running", "4", "--ignore-eos"]
    res = subprocess.run(cmd, capture_output=True, text=True, cwd=str(util.ROOT), timeout=600)
    assert res.returncode == 0, res.stderr
    rows = [json.loads(line) for line in res.stdout.strip().splitlines() if line.startswith("{")]
    for row, prompt in zip(rows, ([5, 17, 3], [9, 8, 7, 6, 11, 2])):
        want, gaps = VP.greedy(plain_cfg, w, prompt, 6)
        for a, b, gap in zip(row["token_ids"], want, gaps):
            if gap < 1e-3:
                break
            assert a == b, f"the command line generated {row['token_ids']}, the plain implementation {want}"
    assert len(rows) == 2


def test_bfloat16_generation_with_graphs_equals_eager(tmp_path):
    from oxr_inference_b200.config import EngineSettings
    from oxr_inference_b200.engine.api import Engine, SamplingParams

    cfg = VU.MODEL_C
    folder = VU.make_folder(tmp_path, cfg, "C", seed=12)
    prompts = [VU.tokens(cfg, n, seed=40 + n) for n in (17, 3, 30, 8)]
    out = []
    for graphs in (False, True):
        engine = Engine(folder, EngineSettings(dtype="bfloat16", num_pages=48, page_size=16, max_running=4, cuda_graphs=graphs))
        out.append([c.token_ids for c in engine.generate(prompts, SamplingParams(max_tokens=10, ignore_eos=True))])
    assert out[0] == out[1]


# ------------------------------------------------------------------------------------------------ marked keys: windows and maps alone
def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def plain_attention(q, k, v, pos, window):
    """One request: q [n, H, D] at positions pos, keys / values [ctx, KV, D] (fp64), scores q . k."""
    per = q.shape[1] // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(per, 1))
    j = torch.arange(k.shape[0])
    seen = j[None, :] <= pos[:, None]
    if window > 0:
        seen &= pos[:, None] - j[None, :] < window
    return torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen[None], -math.inf), -1), v.repeat_interleave(per, 1))


def marked_case(dtype, H, G, D, DV, window, q_lens, ctx_lens, marks, P=8):
    """Differential attention from projections to the combined heads, with the cache filled by the kernel itself: requests whose keys are small but
    for one MARKED key each, which map 1 of every head points at and map 2 points away from. Where the mark is visible map 1 is that key's
    value and map 2 an average of the others; where it is not, both are averages. Pages are dealt out in a shuffled order."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(H * 1000 + D + window * 7)
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    size = (max(2 * D, DV) + 15) // 16 * 16
    tiled = ops.tiled_attention_takes(size, size, tdt)
    W, WV = (size, size) if tiled else (2 * D, DV)
    n_pages = sum(-(-c // P) for c in ctx_lens) + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    k_pool, v_pool = torch.zeros(n_pages, P, G, W, dtype=tdt, device=DEV), torch.zeros(n_pages, P, G, WV, dtype=tdt, device=DEV)
    table = torch.full((len(ctx_lens), max(-(-c // P) for c in ctx_lens)), -1, dtype=torch.int32)
    direction = torch.randn(D, generator=g)
    direction = direction / direction.norm()
    bias = torch.randn(2 * H * D + 2 * G * D + G * DV, generator=g) * 0.3
    lam, eps, factor = 0.37, 1e-5, 0.6
    rows, slots, wants, starts = [], [], [], []
    for r, (c, ql, mark) in enumerate(zip(ctx_lens, q_lens, marks)):
        q = torch.randn(c, H, 2, D, generator=g) * 0.3
        q[:, :, 0] += direction * 4.0
        q[:, :, 1] -= direction * 4.0
        k = torch.randn(c, G, 2, D, generator=g) * 0.3
        k[mark] = direction * 6.0
        proj = (torch.cat([q.reshape(c, -1), k.reshape(c, -1), torch.randn(c, G * DV, generator=g)], 1) - bias).to(tdt)
        for j in range(c):
            if j % P == 0:
                table[r, j // P] = order.pop()
            slots.append(int(table[r, j // P]) * P + j % P)
        rows.append(proj)
        starts.append(c - ql)
        full = proj.double() + bias.double()
        qd, kd, vd = full[:, :2 * H * D].reshape(c, H, 2, D), full[:, 2 * H * D:2 * (H + G) * D].reshape(c, G, 2, D), full[:, 2 * (H + G) * D:].reshape(c, G, DV)
        pos = torch.arange(c - ql, c)
        one, two = (plain_attention(qd[c - ql:, :, m], kd[:, :, m], vd, pos, window) for m in (0, 1))
        wants.append((VP.rms(one - lam * two, eps) * factor).reshape(ql, -1))
    status = ops.new_status(DEV)
    q_all = ops.diff_prep(torch.cat(rows).to(DEV), num_heads=H, num_kv_heads=G, dim=D, value_dim=DV, width=W, bias=bias.to(DEV), k_pool=k_pool, v_pool=v_pool,
                          slots=i32(slots), status=status)
    base, keep = 0, []
    for c, ql in zip(ctx_lens, q_lens):
        keep += list(range(base + c - ql, base + c))
        base += c
    q_new = q_all[torch.tensor(keep, device=DEV)].contiguous()
    if tiled:
        maps = ops.make_kv_maps(k_pool.unsqueeze(0), v_pool.unsqueeze(0), P)
        tiles = {}
        for spec in ops.attention_tile_specs(2 * H, G, W, tdt, P if maps is not None else None):
            treq = [r for r, ql in enumerate(q_lens) if spec[1] <= ql <= spec[2] for _ in range(0, ql, spec[0])]
            ttok = [t0 for r, ql in enumerate(q_lens) if spec[1] <= ql <= spec[2] for t0 in range(0, ql, spec[0])]
            tiles[spec] = (i32(treq or [0]), i32(ttok or [0]), len(treq))
        o = ops.paged_attention(q_new.view(-1, 2 * H, W), k_pool, v_pool, tiles=tiles, cu_q=i32([0] + torch.tensor(q_lens).cumsum(0).tolist()),
                                ctx_lens=i32(ctx_lens), block_table=table.to(DEV), page_size=P, scale=1.0, window=window, kv_len_bound=max(ctx_lens),
                                status=status, kv_maps=maps)
    else:
        positions = i32([p for s, ql in zip(starts, q_lens) for p in range(s, s + ql)])
        req_of = i32([r for r, ql in enumerate(q_lens) for _ in range(ql)])
        o = ops.attention_rows(q_new, 2 * H, k_pool, v_pool, value_dim=DV, positions=positions, req_of_token=req_of, block_table=table.to(DEV), scale=1.0,
                               window=window, status=status).view(-1, 2 * H, DV)
    got = ops.diff_combine(o, H, DV, torch.tensor([lam], device=DEV), eps, factor)
    ops.check_status(status)
    want = torch.cat(wants).float()
    err = (got.float().cpu() - want).abs().max() / want.abs().max()
    assert err < (3e-5 if dtype == "float32" else 4e-2), f"off by {err:.2e} of the largest entry"


WINDOW = 21


# the marked key: far back (outside the window), just outside and just inside it for the last token, on a page's first and last row, the query itself
@pytest.mark.parametrize("mark", [0, 7, 8, 129 - WINDOW, 130 - WINDOW, 119, 120, 128, 129])
@pytest.mark.parametrize("dtype,H,G,D,DV", [("float32", 3, 1, 10, 24), ("bfloat16", 6, 2, 32, 64), ("bfloat16", 2, 2, 24, 16), ("bfloat16", 4, 1, 64, 128)])
def test_marked_keys_inside_and_outside_the_window_of_both_maps(dtype, H, G, D, DV, mark):
    marked_case(dtype, H, G, D, DV, WINDOW, [70, 1, 5, 2], [130, 130, 130, 2], [mark, mark, mark, 0])
    marked_case(dtype, H, G, D, DV, 0, [70, 1, 5, 2], [130, 130, 130, 2], [mark, mark, mark, 0])


# ------------------------------------------------------------------------------------------------ the new kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,DIM", [(3, 12), (2, 16), (2, 30), (2, 48), (3, 64), (2, 70), (2, 128), (1, 200), (1, 256)])
def test_delta_scan_continues_from_its_state(dtype, H, DIM):
    """Two requests in unequal portions over four steps (portions beside a single token, twice single tokens alone, portions again) against the
    recurrence in float64, token by token; the state a step leaves is the state the next one starts from; a slot nobody uses stays zero."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(H + DIM)
    lens, inner, lead = [41, 11], H * DIM, 8
    ins = [(torch.randn(n, 4 * inner + lead, generator=g).to(dtype), torch.randn(n, inner + 5, generator=g), torch.randn(n, inner, generator=g)) for n in lens]
    w0, ab = torch.randn(inner, generator=g) - 1.0, torch.randn(inner, generator=g)
    state = torch.zeros(4, lead + inner * DIM, device=DEV)[:, lead:]       # a view with a row stride of its own
    got, at = [[], []], [0, 0]
    for cut in ([29, 1], [1, 1], [1, 1], [10, 8]):
        parts, cu = [[], [], []], [0]
        for r in (0, 1):
            for p, x in zip(parts, ins[r]):
                p.append(x[at[r]:at[r] + cut[r]])
            cu.append(cu[-1] + cut[r])
        proj, za, zw = (torch.cat(p).to(DEV) for p in parts)
        y = ops.delta_scan(proj, lead, lead + inner, lead + 2 * inner, zw, w0.to(DEV), za, ab.to(DEV), heads=H, key_dim=DIM, value_dim=DIM, rate=math.exp(-0.5),
                           len_eps=1e-6, state=state, cu_q=i32(cu), state_slots=i32([2, 0]), n_requests=2, single_tokens=cut == [1, 1])
        for r in (0, 1):
            got[r].append(y[cu[r]:cu[r + 1]].cpu())
            at[r] += cut[r]
    for r, n in enumerate(lens):
        p, heads = ins[r][0].double()[:, lead:], lambda x: x.reshape(n, H, DIM)
        decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(ins[r][2].double() + w0.double()))
        rate = torch.sigmoid(ins[r][1][:, :inner].double() + ab.double())
        want = VP.delta_rule(heads(p[:, :inner]), heads(p[:, inner:2 * inner]), heads(p[:, 2 * inner:3 * inner]), heads(decay), heads(rate))
        err = (torch.cat(got[r]).double().reshape(n, H, DIM) - want).abs().max() / want.abs().max()
        assert err < 2e-5, f"request {r}: off by {err:.2e}"
    assert state[1].abs().max() == 0 and state[3].abs().max() == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,rows", [(52, 0), (64, 1), (1032, 3), (1000, 4), (4104, 2), (8200, 0)])
def test_shift_norm_continues_from_its_state(dtype, hidden, rows):
    """Three requests in unequal portions (one sits a step out) with and without a pending add, against the formulas; blocks of several rows that
    begin inside a request, at its first token and before it."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(hidden + rows)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lens = [23, 9, 14]
    streams, ys = [rnd(n, hidden) for n in lens], [(2 * rnd(n, hidden)).to(dtype) for n in lens]
    w, post, mu, eps, post_eps = 1 + 0.1 * rnd(hidden), 1 + 0.1 * rnd(hidden), 0.5 + 0.3 * rnd(hidden), 1e-5, 1e-4
    slots = [3, 0, 1]
    for pending in (False, True):
        state = torch.zeros(5, 4 + hidden, device=DEV)[:, 4:]
        at, got, news = [0, 0, 0], [[], [], []], [[], [], []]
        for cut in ([2, 1, 5], [1, 1, 1], [13, 0, 6], [7, 7, 2]):
            live = [r for r in range(3) if cut[r]]
            cu = [0]
            for r in live:
                cu.append(cu[-1] + cut[r])
            part = lambda xs: torch.cat([xs[r][at[r]:at[r] + cut[r]] for r in live]).to(DEV)
            stream = part(streams)
            before = stream.clone()
            kw = dict(y=part(ys), post_weight=post.to(DEV), post_eps=post_eps) if pending else {}
            out, new = ops.shift_norm(stream, w.to(DEV), eps, mu.to(DEV), state, dtype, req_of_token=i32([i for i, r in enumerate(live) for _ in range(cut[r])]),
                                      cu_q=i32(cu), state_slots=i32([slots[r] for r in live]), rows_per_block=rows, **kw)
            assert torch.equal(stream, before), "the stream that is read stays as it was"
            for i, r in enumerate(live):
                got[r].append(out[cu[i]:cu[i + 1]].double().cpu())
                news[r].append(new[cu[i]:cu[i + 1]].double().cpu())
                at[r] += cut[r]
        tol = 2e-5 if dtype == torch.float32 else 2e-2
        for r in range(3):
            s = streams[r].double() + (VP.rms(ys[r].double(), post_eps) * post.double() if pending else 0.0)
            h = VP.rms(s, eps) * w.double()
            want = VP.token_shift(h, mu.double())
            assert (torch.cat(news[r]) - s).abs().max() < 2e-5 * (1 + s.abs().max()), f"stream of request {r}"
            assert (torch.cat(got[r]) - want).abs().max() < tol * (1 + want.abs().max()), f"request {r}, pending {pending}"
            assert (state[slots[r]].double().cpu() - h[-1]).abs().max() < 2e-5 * (1 + h[-1].abs().max()), f"state of request {r}"
        assert state[2].abs().max() == 0 and state[4].abs().max() == 0


def near(got, want, tol, what):
    err = float((got.double().cpu() - want).abs().max() / (1 + want.abs().max()))
    assert err <= tol, f"{what}: off by {err:.2e}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,rank,rot,dim,lead", [(3, 24, 8, 12, 28), (4, 64, 32, 32, 32), (5, 192, 64, 128, 1024), (2, 13, 6, 7, 11), (1, 16, 16, 8, 8)])
def test_latent_rows_and_queries_with_half_split_pairs(dtype, H, rank, rot, dim, lead):
    """The queries' latent (columns of a wider product, normed), the cache row and the rotated parts, against the formulas; the row of a token that is
    not stored stays as it was."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(H + rank)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    n = 37
    both, q = rnd(n, lead + rank + rot).to(dtype), rnd(n, H, dim + rot).to(dtype)
    wq, wc, eps = 1 + 0.1 * rnd(lead), 1 + 0.1 * rnd(rank), 1e-5
    dev = both.to(DEV)
    near(ops.cols_rms_norm(dev[:, :lead], wq.to(DEV), eps), VP.rms(both[:, :lead].double(), eps) * wq.double(), tol, "queries' latent")
    ang = torch.arange(n, dtype=torch.float64)[:, None] * torch.tensor([30.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    pool, q_abs = torch.zeros(6, 8, 1, rank + rot, dtype=dtype, device=DEV), torch.zeros(n, H, rank + rot, dtype=dtype, device=DEV)
    slots = torch.randperm(48, generator=g)[:n].tolist()
    slots[5] = -1
    status = ops.new_status(DEV)
    ops.latent_prep(pool, dev[:, lead:], rank, rot, wc.to(DEV), eps, q.to(DEV), H, dim + rot, dim, q_abs, rank + rot, rank, ang.cos().float().to(DEV),
                    ang.sin().float().to(DEV), i32(slots), status, halves=True)
    ops.check_status(status)
    down = both[:, lead:].double()
    row = torch.cat([VP.rms(down[:, :rank], eps) * wc.double(), VP.rotate_halves(down[:, None, rank:], rot, 30.0)[:, 0]], 1)
    keep = [t for t in range(n) if t != 5]
    flat = pool.view(48, -1)
    near(flat[torch.tensor(slots, device=DEV)[keep]], row[keep], tol, "cache rows")
    assert sum(bool(flat[s].abs().max() > 0) for s in range(48)) == n - 1
    near(q_abs[:, :, rank:], VP.rotate_halves(q[:, :, dim:].double(), rot, 30.0), tol, "rotated queries")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 8, 13, 16, 17, 130])
@pytest.mark.parametrize("H,n_in,n_out", [(3, 12, 24), (2, 64, 192), (4, 16, 80), (2, 13, 7), (5, 192, 128)])
def test_per_head_maps(dtype, n, H, n_in, n_out):
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(n + n_in)
    x, w = torch.randn(n, H, n_in + 8, generator=g).to(dtype), (torch.randn(H, n_in, n_out, generator=g) * n_in ** -0.5).to(dtype)
    out = torch.full((n, H, n_out + 16), 7.0, dtype=dtype, device=DEV)
    ops.head_linear(out, 8, x.to(DEV), 8, w.to(DEV))
    near(out[:, :, 8:8 + n_out], torch.einsum("thi,hio->tho", x[:, :, 8:].double(), w.double()), 2e-5 if dtype == torch.float32 else 1e-2, "per-head map")
    assert (out[:, :, :8] == 7).all() and (out[:, :, 8 + n_out:] == 7).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,KV,DK,half,after,n", [(6, 2, 64, 16, False, 70), (20, 4, 128, 32, False, 66), (20, 4, 128, 64, True, 5), (18, 6, 64, 0, True, 80), (5, 5, 24, 12, False, 70)])
def test_head_prep_with_a_factor_per_query_head(dtype, H, KV, DK, half, after, n):
    """Bias, norm, rotation and a factor per head, for steps of many and of few tokens (different kernels), against float64."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(H + DK + n)
    rnd = lambda *s: torch.randn(*s, generator=g)
    cq, ck = H * DK, KV * DK
    proj, bias, factor = rnd(n, cq + 2 * ck).to(dtype), rnd(cq + ck), 1 + rnd(H)
    qw, kw, eps = 1 + 0.2 * rnd(DK), 1 + 0.2 * rnd(DK), 1e-5
    k_pool, v_pool = (torch.zeros(12, 8, KV, DK, dtype=dtype, device=DEV) for _ in range(2))
    slots = torch.randperm(96, generator=g)[:n]
    cos = sin = None
    if half:
        ang = torch.arange(n, dtype=torch.float64)[:, None] * torch.tensor([40.0 ** (-i / half) for i in range(half)], dtype=torch.float64)
        cos, sin = ang.cos().float().to(DEV), ang.sin().float().to(DEV)
    status = ops.new_status(DEV)
    q = ops.head_prep(proj.to(DEV), q_col0=0, k_col0=cq, v_col0=cq + ck, num_heads=H, num_kv_heads=KV, key_dim=DK, value_dim=DK, bias=bias.to(DEV), norm="weighted",
                      norm_after_rotation=after, q_weight=qw.to(DEV), k_weight=kw.to(DEV), q_factor=factor.to(DEV), eps=eps, cos=cos, sin=sin, k_pool=k_pool,
                      v_pool=v_pool, slots=slots.int().to(DEV), req_of_token=torch.zeros(n, dtype=torch.int32, device=DEV), cu_q=i32([0, n]), state_slots=i32([0]),
                      n_requests=1, status=status)
    ops.check_status(status)

    def steps(x, w):
        turn = (lambda t: VP.rotate_halves(t, 2 * half, 40.0)) if half else (lambda t: t)
        return VP.rms(turn(x), eps) * w.double() if after else turn(VP.rms(x, eps) * w.double())
    full = proj.double()
    full[:, :cq + ck] += bias.double()
    tol = 3e-5 if dtype == torch.float32 else 2.5e-2
    near(q.view(n, H, DK), steps(full[:, :cq].reshape(n, H, DK), qw) * factor.double()[:, None], tol, "queries")
    near(k_pool.view(96, KV, DK)[slots.to(DEV)], steps(full[:, cq:cq + ck].reshape(n, KV, DK), kw), tol, "keys")
    near(v_pool.view(96, KV, DK)[slots.to(DEV)], full[:, cq + ck:].reshape(n, KV, DK), tol, "values")


@pytest.mark.parametrize("E,identity,top,groups,keep", [(7, 2, 3, 1, 1), (20, 4, 4, 1, 1), (5, 0, 5, 1, 1), (24, 8, 6, 4, 2), (300, 20, 9, 1, 1), (40, 10, 4, 1, 1)])
def test_router_with_corrections_and_identity_experts(E, identity, top, groups, keep):
    """The choice by score + correction (which may be negative), the weights of the bare scores, and the identity experts' sum; E > 256 takes the
    kernel with a thread per token."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(E + top)
    n = 19
    z, corr = torch.randn(n, E, generator=g) * 2, torch.randn(E, generator=g) - 1.5
    kept = torch.empty(n, device=DEV)
    gate, ids, wts = ops.route(z.to(DEV), top=top, groups=groups, keep=keep, scale=1.3, score="softmax", group_score="max", renormalize=False,
                               correction=corr.to(DEV), kept=kept, identity=identity)
    s = torch.softmax(z.double(), -1)
    c = s + corr.double()
    if groups > 1:
        best = torch.topk(c.reshape(n, groups, -1).amax(-1), keep, -1).indices
        allowed = torch.zeros(n, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(E // groups, 1)
        c = c.masked_fill(~allowed, -math.inf)
    want = torch.topk(c, top, -1).indices
    assert torch.equal(ids.cpu().long(), want)
    w = torch.gather(s, 1, want) * 1.3
    near(wts, w, 2e-6, "weights")
    dense = torch.zeros(n, E, dtype=torch.float64).scatter_(1, want, w)
    assert gate.shape == (n, E - identity)
    near(gate, dense[:, :E - identity], 2e-6, "dense row")
    if identity:
        near(kept, dense[:, E - identity:].sum(-1), 2e-6, "identity experts")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_small_kernels_against_their_formulas(dtype):
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for n, inter, k, inner in ((5, 24, 16, 0), (40, 32, 64, 8), (3, 9, 16, 0), (130, 64, 72, 8)):
        # the GELU-gated unit: alone, and as the epilogue of a product whose rows alternate in groups of 8
        gu = (2 * rnd(n, 2 * inter)).to(dtype)
        if inner:
            pairs = gu.double().reshape(n, -1, 2, inner)
            gate, up = pairs[:, :, 0].reshape(n, -1), pairs[:, :, 1].reshape(n, -1)
        else:
            gate, up = gu.double()[:, :inter], gu.double()[:, inter:]
        near(ops.gelu_glu(gu.to(DEV), inner), VP.gelu_tanh(gate) * up, tol, "gelu_glu")
        x, w = rnd(n, k).to(dtype), (rnd(2 * inter, k) * 3 * k ** -0.5).to(dtype)
        prod = x.double() @ w.double().T
        p = prod.reshape(n, -1, 2, inner) if inner else torch.stack([prod[:, :inter], prod[:, inter:]], 1)[:, None]
        near(ops.gated_linear(x.to(DEV), w.to(DEV), inner, kind="gelu"), (VP.gelu_tanh(p[:, :, 0]) * p[:, :, 1]).reshape(n, -1), tol, "gated product")
    a, b = rnd(7, 33).to(dtype), rnd(7, 33).to(dtype)
    near(ops.scaled_sum(a.clone().to(DEV), b.to(DEV), 0.7, -1.3), 0.7 * a.double() - 1.3 * b.double(), tol, "scaled_sum")
    z = rnd(9, 30) * 2
    near(ops.tanh_cols(z.to(DEV), 6, 11, dtype), torch.tanh(z[:, 6:17].double()), tol, "tanh_cols")
    # the experts' results with the identity experts' share
    y, place, wts, x, kept = rnd(12, 20).to(dtype), torch.randperm(12, generator=g).int(), torch.rand(4, 3, generator=g), rnd(4, 20).to(dtype), torch.rand(4, generator=g)
    place[[2, 7]] = -1
    want = kept.double()[:, None] * x.double()
    for t in range(4):
        for j in range(3):
            if place[3 * t + j] >= 0:
                want[t] += wts[t, j].double() * y[place[3 * t + j]].double()
    near(ops.combine_rows(y.to(DEV), place.to(DEV), wts.to(DEV), x.to(DEV), kept.to(DEV)), want, tol, "combine_rows")
    near(ops.add_row_gated_(x.clone().to(DEV), y[:4].contiguous().to(DEV), kept.to(DEV), raw=True), x.double() + kept.double()[:, None] * y[:4].double(), tol, "raw row weights")
    # the difference of two maps: heads of one word a lane, of several, and of more than the registers keep
    for H, DV, W in ((3, 11, 16), (2, 128, 128), (2, 200, 208), (1, 1040, 1040), (1, 300, 304)):
        o, lam = rnd(6, 2 * H, W).to(dtype), 0.45
        d = o[:, 0::2, :DV].double() - lam * o[:, 1::2, :DV].double()
        near(ops.diff_combine(o.to(DEV), H, DV, torch.tensor([lam], device=DEV), 1e-5, 0.7), (VP.rms(d, 1e-5) * 0.7).reshape(6, -1), tol, "diff_combine")
