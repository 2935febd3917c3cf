"""Finolix on the GPU against the plain statement in ``tests/plain/finolix_plain.py``: each mechanism alone, the streams' sum after every layer,
whole prompts against token-by-token decoding, portions down to two tokens, batches of unequal requests, pages and slots that are used
again, marked keys far back, at page borders and just inside and outside a window, long decoding, greedy generation through the engine, and
the new kernels against their formulas."""

import math

import pytest
import torch

import finolix_util as FU
from plain import finolix_plain as FP
from util import Replay

pytestmark = pytest.mark.gpu

DEV = "cuda"

CLOSE_CALL = 0.08
"""bfloat16 rows at which some router of the plain model decided by less than this (a difference of logits) are not compared: a logit that
differs by a rounding step may choose another expert there, for no fault. (32-bit compares every row.)"""


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
L, G, MOE, DENSE, CFG = FU.latent, FU.gated, FU.moe, FU.dense, FU.model_config
SINGLE = {
    "latent_alone": CFG([L()]),
    "latent_one_head_two_rotated_entries": CFG([L(heads=1, rot_dim=2, dim=4, kv_rank=16, q_rank=8)]),
    "latent_tiled_sizes": CFG([L(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=32, size=19)], width=64),
    "latent_tiled_sizes_three_heads": CFG([L(heads=3, dim=16, rot_dim=8, vdim=48, kv_rank=40, q_rank=24, size=9)], width=64),
    "latent_odd_sizes": CFG([L(heads=3, dim=7, rot_dim=6, vdim=9, kv_rank=13, q_rank=11)], width=39),
    "latent_wide_row": CFG([L(heads=2, dim=32, rot_dim=32, vdim=16, kv_rank=256, q_rank=48, scale=0.2)]),
    "latent_window_of_one": CFG([L(size=1)]),
    "latent_window_of_a_page": CFG([L(size=8, heads=4, kv_rank=56, q_rank=16)]),
    "latent_window_beyond_the_prompt": CFG([L(size=500)]),
    "latent_without_scaling": CFG([L(scaling=None)]),
    "latent_ramp_within_one_pair": CFG([L(scaling=FU.ramp(3.0, 30, 2.0, 1.9))]),
    "gated_alone": CFG([G()]),
    "gated_equal_sizes_all_rotated": CFG([G(heads=6, kv_heads=3, dim=32, vdim=32, rot=32, scale=0.2)], width=64),
    "gated_two_rotated_entries": CFG([G(rot=2, base=5.0)]),
    "gated_values_wider_than_keys": CFG([G(heads=5, kv_heads=1, dim=8, vdim=64, rot=4)]),
    "gated_odd_sizes": CFG([G(heads=3, kv_heads=1, dim=7, vdim=11, rot=6)], width=39),
    "gated_tma_sizes": CFG([G(heads=6, kv_heads=3, dim=64, vdim=64, rot=16, scale=0.15)], width=64),
    "one_stream": CFG([L(mlp=DENSE()), G(mlp=DENSE(ff=24))], streams=1),
    "two_streams": CFG([L(mlp=DENSE()), G(mlp=DENSE(ff=24))], streams=2, width=64),
    "four_streams": CFG([L(mlp=DENSE()), G(mlp=DENSE(ff=24))], streams=4, width=64),
    "seven_streams": CFG([L(mlp=DENSE()), G(mlp=DENSE(ff=24))], streams=7),
    "dense_feed_forward": CFG([G(mlp=DENSE())]),
    "dense_feed_forward_odd": CFG([G(mlp=DENSE(ff=29))], width=39),
    "dense_feed_forward_wide": CFG([G(mlp=DENSE(ff=96))], width=64),
    "experts": CFG([G(mlp=MOE())]),
    "experts_top_one": CFG([G(mlp=MOE(experts=6, top=1))]),
    "experts_all_chosen": CFG([G(mlp=MOE(experts=4, top=4, ff=20))]),
    "one_expert": CFG([G(mlp=MOE(experts=1, top=1))]),
    "experts_odd_sizes": CFG([G(mlp=MOE(experts=7, top=3, ff=9))], width=39),
    "one_layer_three_times": CFG([L(mlp=DENSE(ff=24)), FU.again([L(mlp=DENSE(ff=24))], 0), FU.again([L(mlp=DENSE(ff=24))], 0)]),
    "weights_of_a_later_layer": CFG([{**G(), "weights_of": 1}, G()]),
    "no_feed_forward_between_layers_that_have_one": CFG([L(mlp=DENSE()), G(), L(), G(mlp=DENSE(ff=24))]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_mechanism(name, dtype, tmp_path):
    cfg = SINGLE[name]
    folder = FU.make_folder(tmp_path, cfg, name, seed=5)
    ids = FU.tokens(cfg, 61, seed=1)
    want = FU.plain_logits(folder, ids)
    r = runner_for(folder, dtype)
    mg = FU.router_margins(folder, ids)
    close(run_cut(r, ids, [61]), want, dtype, f"{name}, whole prompt", mg)
    close(run_cut(r, ids, [29] + [1] * 32), want, dtype, f"{name}, 29 tokens then one by one", mg)
    close(run_cut(r, ids, [2, 3, 2, 11, 2, 17, 1, 2, 21]), want, dtype, f"{name}, portions", mg)


@pytest.mark.parametrize("width,ff,experts,top", [(64, 16, 6, 2), (40, 20, 5, 3), (72, 36, 3, 2), (39, 9, 4, 3)])
def test_experts_grouped_by_expert_equal_the_two_products_form(width, ff, experts, top, tmp_path):
    """From ``grouped_min_rows`` tokens on every expert multiplies only the rows that chose it; below, all experts are two products. Both
    against the plain sum, in both dtypes, also for odd widths."""
    cfg = CFG([G(mlp=MOE(experts=experts, top=top, ff=ff))], width=width)
    folder = FU.make_folder(tmp_path, cfg, "grouped", seed=8)
    ids = FU.tokens(cfg, 70, seed=3)
    want, mg = FU.plain_logits(folder, ids), FU.router_margins(folder, ids)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(folder, dtype)
        part = r.model.blocks[0].feed_forward
        for rows in (0, 8):
            part.grouped_min_rows = rows
            close(run_cut(r, ids, [40, 5, 25]), want, dtype, f"experts, grouped from {rows} rows on, {dtype}", mg)


def test_layer_results_one_by_one(tmp_path):
    """The sum of the streams after every layer against the plain statement's, in 32-bit (a layer's last update is still pending when it returns)."""
    from oxr_inference_b200.engine.batch import StepEntry

    for name, cfg in (("A", FU.MODEL_A), ("B", FU.MODEL_B)):
        folder = FU.make_folder(tmp_path, cfg, name, seed=2)
        ids = FU.tokens(cfg, 23, seed=6)
        plain_cfg, w = FP.read_model(folder, torch.float64)
        want: list = []
        FP.forward(plain_cfg, w, ids, streams=want)
        r = runner_for(folder, "float32")
        got = []
        for b in r.model.blocks:
            def wrapped(*a, _f=b.forward, **k):
                out = _f(*a, **k)
                got.append(out[1].clone() if out[0] is None else out[0].total(out[1]))
                return out
            b.forward = wrapped
        rc = r.cache.open("r")
        assert r.cache.reserve(rc, len(ids))
        r.step([StepEntry(rc, ids, [len(ids) - 1])])
        r.cache.close(rc)
        assert len(got) == len(want) == len(cfg["layers"])
        for i, (a, b) in enumerate(zip(got, want)):
            err = (a.double().cpu() - b).abs().max() / b.abs().max()
            assert err < 2e-5, f"model {name}, layer {i} ({cfg['layers'][i]['type']}): off by {err:.2e} of the sum's largest entry"


# ------------------------------------------------------------------------------------------------ whole models, every cutting
MODELS = {"A": FU.MODEL_A, "B": FU.MODEL_B, "C": FU.MODEL_C}
SPREADING = {"A": True, "B": True, "C": False}
"""Whether a model has routers below attention layers (see ``close``)."""


@pytest.fixture(scope="module", params=[(m, d) for m in sorted(MODELS) for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def model(request, tmp_path_factory):
    name, dtype = request.param
    # 32-bit runs take the weights at full strength and compare every row at 2e-4; 16-bit runs of these deep models take them milder
    folder = FU.make_folder(tmp_path_factory.mktemp(f"finolix_{name}_{dtype}"), MODELS[name], name, seed=11, strength=1.0 if dtype == "float32" else 0.25)
    return name, dtype, folder, runner_for(folder, dtype, page_size=8, num_pages=40)


def test_whole_prompt_equals_token_by_token(model):
    name, dtype, folder, r = model
    cfg = MODELS[name]
    for n in (1, 2, 9, 75):
        ids = FU.tokens(cfg, n, seed=2)
        want, mg = FU.plain_logits(folder, ids), FU.router_margins(folder, ids)
        close(run_cut(r, ids, [n]), want, dtype, f"{name}: whole prompt of {n}", mg, SPREADING[name])
        close(run_cut(r, ids, [1] * n), want, dtype, f"{name}: {n} tokens one by one", mg, SPREADING[name])


def test_portions_of_several_sizes(model):
    name, dtype, folder, r = model
    ids = FU.tokens(MODELS[name], 120, seed=3)
    want, mg = FU.plain_logits(folder, ids), FU.router_margins(folder, ids)
    for cuts in ([2] * 60, [7, 2, 13, 3, 2, 31, 1, 16, 2, 17, 8, 18], [33, 33, 33, 21], [119, 1], [15, 16, 17, 32, 40]):
        close(run_cut(r, ids, cuts), want, dtype, f"{name}: portions {cuts[:4]}...", mg, SPREADING[name])


def test_long_decoding(model):
    name, dtype, folder, r = model
    ids = FU.tokens(MODELS[name], 260, seed=4)
    close(run_cut(r, ids, [4] + [1] * 256), FU.plain_logits(folder, ids), dtype, f"{name}: 256 decoded tokens", FU.router_margins(folder, ids), SPREADING[name])


def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(model):
    """Four live requests at most, 40 pages of 8 tokens: the lengths below need far more over time, so pages and state slots come back and are
    handed out again; every request's logits equal those it gets alone."""
    name, dtype, folder, r = model
    cfg = MODELS[name]
    lengths = [97, 3, 64, 30, 1, 121, 45, 18, 70]
    todo = [(f"q{i}", FU.tokens(cfg, n, seed=20 + i)) for i, n in enumerate(lengths)]
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
        ids = FU.tokens(cfg, n, seed=20 + i)
        mixed = torch.cat(got[f"q{i}"])
        if dtype == "bfloat16" and SPREADING[name]:
            # what the mix must not change is told apart from what 16 bits do to a deep model with routers: the same request alone, cut alike
            alone = run_cut(r, ids, cuts[f"q{i}"]).float().cpu()
            d = (mixed.float().cpu() - alone) - (mixed.float().cpu() - alone).mean(-1, keepdim=True)
            err = d.pow(2).mean(-1).sqrt() / alone.std(-1).clamp_min(1e-6)
            assert int((err > 3e-2).sum()) <= n // 20, f"{name}: request {i} of {n} tokens differs in the mix from itself alone: row {int(err.argmax())} by {err.max():.2e}"
        else:
            close(mixed, FU.plain_logits(folder, ids), dtype, f"{name}: request {i} of {n} tokens in the mix", FU.router_margins(folder, ids))


def test_far_keys(tmp_path):
    """A prompt of 700 tokens with peaked attention: the last logits rest on keys from hundreds of tokens back, across dozens of pages; in 32-bit a
    lost key shows."""
    cfg = CFG([L(heads=4, dim=16, rot_dim=16, vdim=32, kv_rank=48, q_rank=32, size=300, base=1e4, scaling=FU.ramp(8.0, 100, 16.0, 1.0), mlp=DENSE(ff=40)),
               G(heads=2, kv_heads=1, dim=64, vdim=64, rot=32, base=1e4, scale=0.2),
               G(heads=4, kv_heads=2, dim=16, vdim=32, rot=4, base=1e5, scale=0.5, mlp=MOE(ff=16, experts=4, top=2))], width=64, vocab=180, streams=2)
    ids = FU.tokens(cfg, 700, seed=9)
    for dtype in ("float32", "bfloat16"):        # the model's router stands in its last layer; 16-bit runs take the weights milder, as above
        folder = FU.make_folder(tmp_path, cfg, f"far_{dtype}", seed=3, sharpen=4.0, strength=1.0 if dtype == "float32" else 0.25)
        want, mg = FU.plain_logits(folder, ids), FU.router_margins(folder, ids)
        r = runner_for(folder, dtype, page_size=16, num_pages=50)
        close(run_cut(r, ids, [650] + [1] * 50), want, dtype, f"{dtype}: 650 tokens, then 50 one by one", mg)
        close(run_cut(r, ids, [255, 257, 2, 186]), want, dtype, f"{dtype}: portions that end beside page borders", mg)


def test_windows_release_their_pages_and_nothing_else(tmp_path):
    cfg = CFG([L(size=9), G(), L(size=20)])
    r = runner_for(FU.make_folder(tmp_path, cfg, "windows", seed=1), "float32", page_size=4, num_pages=40)
    rc = r.cache.open("r")
    ids = FU.tokens(cfg, 60, seed=1)
    r.step([feed(r, rc, ids, 0, 60)])
    by_window = {g.need.window: sum(p >= 0 for p in rc.tables[i]) for i, g in enumerate(r.cache.plan.groups)}
    assert by_window == {9: 2, 20: 5, 0: 15}      # the next query sits at 60 and sees keys from 52, from 41 and from 0 on
    r.cache.close(rc)
    r.cache.check()


def test_replay_program_runs_the_design(tmp_path):
    cfg = FU.MODEL_A
    folder = FU.make_folder(tmp_path, cfg, "A", seed=11)
    ids_a, ids_b = FU.tokens(cfg, 50, seed=7), FU.tokens(cfg, 9, seed=8)
    r = Replay(folder, "float32", tmp_path / "out", max_tokens=128, page_size=16)
    got = r.step([{"id": "a", "tokens": ids_a[:31], "want": [0, 30]}, {"id": "b", "tokens": ids_b[:2], "want": []}])
    close(got, FU.plain_logits(folder, ids_a)[[0, 30]], "float32", "replay: first step")
    assert r.step([{"id": "b", "tokens": ids_b[2:8], "want": []}]) is None
    got = r.step([{"id": "a", "tokens": ids_a[31:], "want": [18]}, {"id": "b", "tokens": ids_b[8:], "want": [0]}], end=["a", "b"])
    close(got, torch.stack([FU.plain_logits(folder, ids_a)[49], FU.plain_logits(folder, ids_b)[8]]), "float32", "replay: last step")
    assert r.close() == 0


# ------------------------------------------------------------------------------------------------ greedy generation through the engine
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_engine(which, graphs, tmp_path):
    from oxr_inference_b200.config import EngineSettings
    from oxr_inference_b200.engine.api import Engine, SamplingParams

    cfg = MODELS[which]
    folder = FU.make_folder(tmp_path, cfg, which, seed=11)
    plain_cfg, w = FP.read_model(folder, torch.float64)
    prompts = [FU.tokens(cfg, n, seed=30 + n) for n in (5, 23, 1, 40, 12, 9)]
    engine = Engine(folder, EngineSettings(dtype="float32", num_pages=48, page_size=8, max_running=3, max_step_tokens=32, prefill_chunk=16,
                                           cuda_graphs=graphs))
    done = engine.generate(prompts, SamplingParams(max_tokens=14, ignore_eos=True))
    compared = 0
    for prompt, c in zip(prompts, done):
        want, gaps = FP.greedy(plain_cfg, w, prompt, 14)
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

    cfg = FU.MODEL_A
    folder = FU.make_folder(tmp_path, cfg, "A", seed=14)
    plain_cfg, w = FP.read_model(folder, torch.float64)
    cmd = [sys.executable, "-m", "oxr_inference_b200", "--model", str(folder), "--prompt-ids", "5,17,3", "--prompt-ids", "9 8 7 6 11 2",
           "--max-tokens", "6", "--dtype", "float32", "--num-pages", "32", "--max-running", "4", "--ignore-eos"]
    res = subprocess.run(cmd, capture_output=True, text=True, cwd=str(util.ROOT), timeout=600)
    assert res.returncode == 0, res.stderr
    rows = [json.loads(line) for line in res.stdout.strip().splitlines() if line.startswith("{")]
    for row, prompt in zip(rows, ([5, 17, 3], [9, 8, 7, 6, 11, 2])):
        want, gaps = FP.greedy(plain_cfg, w, prompt, 6)
        for a, b, gap in zip(row["token_ids"], want, gaps):
            if gap < 1e-3:
                break
            assert a == b, f"the command line generated {row['token_ids']}, the plain implementation {want}"
    assert len(rows) == 2


def test_bfloat16_generation_with_graphs_equals_eager(tmp_path):
    from oxr_inference_b200.config import EngineSettings
    from oxr_inference_b200.engine.api import Engine, SamplingParams

    cfg = FU.MODEL_C
    folder = FU.make_folder(tmp_path, cfg, "C", seed=12)
    prompts = [FU.tokens(cfg, n, seed=40 + n) for n in (17, 3, 30, 8)]
    out = []
    for graphs in (False, True):
        engine = Engine(folder, EngineSettings(dtype="bfloat16", num_pages=48, page_size=16, max_running=4, cuda_graphs=graphs))
        out.append([c.token_ids for c in engine.generate(prompts, SamplingParams(max_tokens=10, ignore_eos=True))])
    assert out[0] == out[1]


# ------------------------------------------------------------------------------------------------ marked keys
def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def plain_rows(q, keys, values, pos, window, sink):
    """[n, H, D] queries at positions ``pos`` over shared rows ``keys [c, D]``, in float64."""
    s = torch.einsum("nhd,cd->nhc", q, keys)
    j = torch.arange(keys.shape[0])
    seen = (j[None] <= pos[:, None]) & ((pos[:, None] - j[None] < window) if window else True)
    s = s.masked_fill(~seen[:, None], -math.inf)
    s = torch.cat([s, sink[None, :, None].expand(s.shape[0], -1, 1)], -1)
    return torch.softmax(s, -1)[..., :-1] @ values


def marked_latent_case(dtype, H, L_, R_, window, q_lens, ctx_lens, marks):
    """Queries of the absorbed form over shared cache rows on scattered pages, with one row per request whose score stands out by far: whether it is
    seen decides the result. The sink is large enough to show as well."""
    from oxr_inference_b200 import ops

    tdt, P, W = getattr(torch, dtype), 8, L_ + R_
    tiled = ops.tiled_attention_takes(W, W, tdt)
    g = torch.Generator().manual_seed(W + H + sum(ctx_lens))
    n_pages = sum(-(-c // P) for c in ctx_lens) + 3
    pool = torch.randn(n_pages, P, 1, W, generator=g).to(tdt).to(DEV)
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((len(ctx_lens), max(-(-c // P) for c in ctx_lens)), -1, dtype=torch.int32)
    direction = torch.randn(W, generator=g)
    direction = direction / direction.norm()
    sink = torch.randn(H, generator=g) + 2.0
    qs, wants, positions, req_of = [], [], [], []
    for r, (c, ql, mark) in enumerate(zip(ctx_lens, q_lens, marks)):
        rows = torch.randn(c, W, generator=g) * 0.3
        rows[mark] = direction * 5.0
        rows = rows.to(tdt)
        for j in range(c):
            if j % P == 0:
                table[r, j // P] = order.pop()
            pool[int(table[r, j // P]), j % P, 0] = rows[j].to(DEV)
        q = (torch.randn(ql, H, W, generator=g) * 0.2 + direction * 3.0).to(tdt)
        pos = torch.arange(c - ql, c)
        wants.append(plain_rows(q.double(), rows.double(), rows[:, :L_].double(), pos, window, sink.double()))
        qs.append(q)
        positions += pos.tolist()
        req_of += [r] * ql
    # a page wholly behind every query's window may have been given back: its entry then names no page
    for r, (c, ql) in enumerate(zip(ctx_lens, q_lens)):
        if window:
            for p in range(max(0, c - ql - window + 1) // P):
                table[r, p] = -1
    status = ops.new_status(DEV)
    q_new = torch.cat(qs).to(DEV)
    if tiled:
        tiles = {}
        for spec in ops.attention_tile_specs(H, 1, W, tdt):
            treq = [r for r, ql in enumerate(q_lens) if spec[1] <= ql <= spec[2] for _ in range(0, ql, spec[0])]
            ttok = [t0 for r, ql in enumerate(q_lens) if spec[1] <= ql <= spec[2] for t0 in range(0, ql, spec[0])]
            tiles[spec] = (i32(treq or [0]), i32(ttok or [0]), len(treq))
        o = ops.paged_attention(q_new, pool, pool, tiles=tiles, cu_q=i32([0] + torch.tensor(q_lens).cumsum(0).tolist()), ctx_lens=i32(ctx_lens),
                                block_table=table.to(DEV), page_size=P, scale=1.0, window=window, kv_len_bound=max(ctx_lens), status=status,
                                sink=sink.to(DEV))[:, :, :L_]
    else:
        o = ops.attention_rows(q_new.view(-1, H * W), H, pool, None, value_dim=L_, positions=i32(positions), req_of_token=i32(req_of),
                               block_table=table.to(DEV), scale=1.0, window=window, sink=sink.to(DEV), status=status).view(-1, H, L_)
    ops.check_status(status)
    want = torch.cat(wants).float()
    err = (o.float().cpu() - want).abs().max() / want.abs().max()
    assert err < (3e-5 if dtype == "float32" else 2e-2), f"off by {err:.2e} of the largest entry"


WINDOW = 21


# the marked row: far back (outside the window), just outside and just inside it for the last token, on a page's first and last row, the query itself
@pytest.mark.parametrize("mark", [0, 7, 8, 129 - WINDOW, 130 - WINDOW, 119, 120, 128, 129])
@pytest.mark.parametrize("dtype,H,L_,R_", [("float32", 3, 24, 8), ("bfloat16", 4, 48, 16), ("bfloat16", 3, 20, 6), ("bfloat16", 20, 112, 16)])
def test_marked_rows_inside_and_outside_the_window_of_latent_attention(dtype, H, L_, R_, mark):
    marked_latent_case(dtype, H, L_, R_, WINDOW, [70, 1, 5, 2], [130, 130, 130, 2], [mark, mark, mark, 0])
    marked_latent_case(dtype, H, L_, R_, 0, [70, 1, 5, 2], [130, 130, 130, 2], [mark, mark, mark, 0])


@pytest.mark.parametrize("back", [0, 149, 150, 151, 1200])
def test_a_small_window_deep_in_a_long_context(back):
    """Single tokens and short portions at 1,500 tokens of context with a window of 150: the split of the keys follows the window, not the context."""
    marked_latent_case("bfloat16", 8, 96, 32, 150, [1, 1, 3, 40], [1500, 700, 1500, 1500], [1499 - back, 699 - min(back, 699), 1497 - back, 1460 - back])


# ------------------------------------------------------------------------------------------------ the new kernels alone
def near(got, want, tol, what):
    err = float((got.double().cpu() - want).abs().max() / (1 + want.abs().max()))
    assert err <= tol, f"{what}: off by {err:.2e}"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,hidden", [(1, 64), (2, 4096), (2, 4104), (3, 1032), (4, 8200), (4, 16400), (2, 39), (5, 64), (16, 50), (4, 13000)])
def test_streams_between_two_sublayers(S, hidden, dtype):
    """Entry from one copy, an update with and without a layer scale, and the way out, against the formulas; the streams are updated in place, except
    where one copy stands for all."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(S + hidden)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n, eps, tol = 5, 1e-5, 3e-5 if dtype == torch.float32 else 1e-2
    x1, y, scale, w = rnd(n, hidden), (2 * rnd(n, hidden)).to(dtype), rnd(hidden), 1 + 0.2 * rnd(hidden)
    mix, outs, ins = rnd(S, S), rnd(S), rnd(S)
    dev = lambda t: t.to(DEV)
    norm = lambda x: FP.rms(FP.read_streams(x, ins.double()), eps) * w.double()
    then = (dev(ins), dev(w), eps)
    h, same = ops.hyper_mix(dev(x1), S, dtype, then=then)
    one = torch.stack([x1.double()] * S)
    near(h, norm(one), tol, "entry")
    near(same, x1.double(), 0.0, "one copy stays one copy")
    for sc in (scale, None):
        ys = y.double() * (sc.double() if sc is not None else 1.0)
        kw = dict(y=dev(y), mix=dev(mix), out_weights=dev(outs), scale=dev(sc) if sc is not None else None)
        want = FP.write_streams(one, mix.double(), outs.double(), ys)
        h, x = ops.hyper_mix(dev(x1), S, dtype, then=then, **kw)
        near(x.transpose(0, 1), want, 3e-6, "streams from one copy")
        near(h, norm(want), tol, "norm behind it")
        again = FP.write_streams(want, mix.double(), outs.double(), ys)
        before = x.clone()
        total = ops.hyper_mix(x, S, dtype, **kw)[1]
        near(total, again.sum(0), 3e-6, "sum of the streams")
        assert torch.equal(x, before), "the way out leaves the streams as they are"
        h, x2 = ops.hyper_mix(x, S, dtype, then=then, **kw)
        assert x2.data_ptr() == x.data_ptr()
        near(x2.transpose(0, 1), again, 3e-6, "streams in place")
        near(h, norm(again), tol, "norm behind the second update")
        near(ops.hyper_mix(dev(x1), S, dtype, **kw)[1], want.sum(0), 3e-6, "sum straight from one copy")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,rank,rot,dim,lead", [(3, 24, 8, 12, 28), (4, 64, 16, 32, 32), (5, 192, 64, 128, 1024), (2, 13, 6, 7, 11), (1, 16, 2, 8, 8), (40, 48, 32, 16, 8)])
def test_latent_rows_and_queries_with_neighbouring_pairs(dtype, H, rank, rot, dim, lead):
    """The cache row and the rotated parts, with angles stretched by a constant, against the formulas; the row of a token that is not stored stays."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(H + rank)
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol, n, eps = 2e-5 if dtype == torch.float32 else 2e-2, 37, 1e-5
    both, q, wc = rnd(n, lead + rank + rot).to(dtype), rnd(n, H, dim + rot).to(dtype), 1 + 0.1 * rnd(rank)
    freq, magnitude = FP.ramp_frequencies(rot, 30.0, FU.ramp())
    cos, sin = ops.rotary_angles(i32(list(range(n))), torch.tensor(freq, dtype=torch.float64, device=DEV), magnitude)
    pool, q_abs = torch.zeros(6, 8, 1, rank + rot, dtype=dtype, device=DEV), torch.zeros(n, H, rank + rot, dtype=dtype, device=DEV)
    slots = torch.randperm(48, generator=g)[:n].tolist()
    slots[5] = -1
    status = ops.new_status(DEV)
    ops.latent_prep(pool, both.to(DEV)[:, lead:], rank, rot, wc.to(DEV), eps, q.to(DEV), H, dim + rot, dim, q_abs, rank + rot, rank, cos, sin, i32(slots), status)
    ops.check_status(status)
    down = both[:, lead:].double()
    row = torch.cat([FP.rms(down[:, :rank], eps) * wc.double(), FP.rotate(down[:, None, rank:], freq, magnitude, True)[:, 0]], 1)
    keep = [t for t in range(n) if t != 5]
    flat = pool.view(48, -1)
    near(flat[torch.tensor(slots, device=DEV)[keep]], row[keep], tol, "cache rows")
    assert sum(bool(flat[s].abs().max() > 0) for s in range(48)) == n - 1
    near(q_abs[:, :, rank:], FP.rotate(q[:, :, dim:].double(), freq, magnitude, True), tol, "rotated queries")
    assert q_abs[:, :, :rank].abs().max() == 0


@pytest.mark.parametrize("E,top,groups,keep", [(7, 3, 1, 1), (5, 5, 1, 1), (1, 1, 1, 1), (24, 6, 4, 2), (300, 9, 1, 1), (64, 8, 1, 1)])
def test_router_with_biases_and_the_softmax_over_the_chosen(E, top, groups, keep):
    """The choice by biased logits, some of them far below the rest, and weights over the chosen alone; E > 256 takes the kernel with a thread per token."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(E + top)
    n = 19
    z, bias = torch.randn(n, E, generator=g) * 3, torch.randn(E, generator=g) * 2
    z[3] -= 200.0
    z[4, ::2] -= 300.0       # exp() of these is zero beside the largest: the order among them still counts
    gate, ids, wts = ops.route(z.to(DEV), top=top, groups=groups, keep=keep, scale=1.0, score="chosen_softmax", group_score="max", bias=bias.to(DEV))
    c = z.double() + bias.double()
    if groups > 1:
        best = torch.topk(c.reshape(n, groups, -1).amax(-1), keep, -1).indices
        allowed = torch.zeros(n, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(E // groups, 1)
        c = c.masked_fill(~allowed, -math.inf)
    want = torch.topk(c, top, -1)
    rows = torch.arange(n) != 3      # a row shifted as a whole loses low bits: near-ties may turn over
    assert torch.equal(ids.cpu().long()[rows], want.indices[rows])
    w = torch.softmax(want.values, -1)
    near(wts[3:4].sum(-1), torch.ones(1, dtype=torch.float64), 1e-6, "a row of very small logits")
    near(wts[rows.to(DEV)], w[rows], 2e-6, "weights")
    near(gate[rows.to(DEV)], torch.zeros(n, E, dtype=torch.float64).scatter_(1, want.indices, w)[rows], 2e-6, "dense row")


@pytest.mark.parametrize("m,n,k", [(1, 40, 24), (8, 96, 64), (16, 33, 72), (9, 64, 39), (40, 200, 64), (100, 4096, 256), (200, 160, 1024), (300, 640, 128), (520, 264, 96),
                                   (1024, 512, 200)])
def test_products_with_the_square_of_relu(m, n, k):
    """Decode-sized products, the sizes between, and the two-SM kernel's, in both dtypes; the plain product of the same sizes stays plain afterwards."""
    from oxr_inference_b200 import ops

    g = torch.Generator().manual_seed(m + n + k)
    for dtype in (torch.float32, torch.bfloat16):
        x, w = torch.randn(m, k, generator=g).to(dtype), (torch.randn(n, k, generator=g) * k ** -0.5).to(dtype)
        z = x.double() @ w.double().T
        near(ops.relu2_linear(x.to(DEV), w.to(DEV)), torch.clamp(z, min=0) ** 2, 1e-5 if dtype == torch.float32 else 1e-2, f"relu2_linear {dtype}")
        near(ops.linear(x.to(DEV), w.to(DEV)), z, 1e-5 if dtype == torch.float32 else 1e-2, f"linear {dtype}")
