"""Sanevik on the GPU: every new kernel form alone against its reference at sizes other than any model's, with
inputs made so that a fault shows (a key that carries all the weight just inside and just outside the window, at
page borders and far back; NaN in pages and slots that belong to nobody); the whole model in float32 and bfloat16
against the plain implementation under every cut of the work; slots and pages used again; long decoding; greedy
generation through ``LLM`` with recorded decode steps; the command line; and ``bin/trace_run`` as a subprocess."""

from __future__ import annotations

import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs as refs
import plain_sanevik as plain
import replay_cases as cases
from fegilix_cases import FakeStep, run_steps
from sanevik_cases import CONFIGS, CONFIG_D, assert_rows_close, oracle as plain_oracle, random_config, write_model
from test_diderax_gpu import DTYPES, ROOT, Arena, Ctx, _rand, _tables, _tol
from tiny_configs import random_prompt

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------ kernels one by one
def _stores(dtype, tables, pages, page, lens, groups, d, dv):
    """Key and value pages with NaN wherever no request has a row."""
    k = torch.full((pages, groups, page, d), float("nan"), dtype=dtype, device="cuda")
    v = torch.full((pages, groups, page, dv), float("nan"), dtype=dtype, device="cuda")
    for b, n in enumerate(lens):
        pos = torch.arange(n)
        where = torch.tensor(tables[b])[pos // page].cuda(), (pos % page).cuda()
        k[where[0], :, where[1]] = _rand(n, groups, d, seed=40 + b, dtype=dtype)
        v[where[0], :, where[1]] = _rand(n, groups, dv, seed=80 + b, dtype=dtype)
    return k, v


@pytest.mark.parametrize("dtype, tensor_cores", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("heads, groups, d, dv, page", [(4, 2, 48, 48, 16), (1, 1, 16, 16, 4), (6, 3, 64, 32, 8), (18, 9, 16, 32, 16), (5, 5, 12, 20, 4),
                                                        (16, 8, 128, 128, 16), (20, 4, 128, 64, 32), (8, 8, 128, 128, 16), (3, 1, 80, 112, 16)])
@pytest.mark.parametrize("window, cap, sink, mixed", [(0, None, True, True), (37, 4.0, False, True), (1, 30.0, False, True), (512, 90.0, True, False),
                                                      (130, 1.0, False, True)])
def test_attention_with_mixed_heads_kernels(dtype, tensor_cores, heads, groups, d, dv, page, window, cap, sink, mixed) -> None:
    """Prompt portions beside single tokens, and steps of single tokens alone (their keys are cut into ranges). The
    caps cover scores far beyond the cap, around it and far below it."""
    from tinyserve_b200.kernels import ops

    if tensor_cores and (d % 16 or dv % 16):
        pytest.skip("sizes of the CUDA-core form")
    talk = _rand(heads, heads, seed=5, scale=0.4).bfloat16().float() if mixed else None
    sinks = _rand(heads, seed=6, scale=2.0) if sink else None
    saved, ops.TALKING_TENSOR_CORES = ops.TALKING_TENSOR_CORES, tensor_cores
    try:
        for lens, news in (([page * 3 + 1, 170, 33, 1, 300], [1, 17, 33, 1, 90]), ([600, 350, 513, 1], [1, 1, 1, 1])):
            tables, table, pages = _tables(lens, page, 7)
            k, v = _stores(dtype, tables, pages, page, lens, groups, d, dv)
            q = _rand(sum(news), heads, d, seed=3, dtype=dtype)
            ctx, res = Ctx(news, lens), []
            for impl in (ops, refs):
                out = torch.full((sum(news), heads * dv), float("nan"), dtype=dtype, device="cuda")
                impl.talking_attention(q, k, v, page, table, ctx, d ** -0.5, window, cap, talk, out, sinks=sinks)
                res.append(out.float())
            scale = float(res[1].abs().max())
            tol = (2e-5 if dtype == torch.float32 else 1e-2) * max(1.0, scale)
            assert not res[0].isnan().any()
            torch.testing.assert_close(res[0], res[1], atol=tol, rtol=0.0)
    finally:
        ops.TALKING_TENSOR_CORES = saved
    if tensor_cores:
        assert ops.talking_cluster(heads, groups, d, dv) > 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("new", [1, 2, 70])
@pytest.mark.parametrize("mixer", ["mixed", "plain"])
@pytest.mark.parametrize("d, page", [(32, 4), (64, 16)])
def test_a_key_just_inside_and_just_outside_the_window(dtype, new, mixer, d, page) -> None:
    """One key outweighs all others for the last query. While it is in the window the output is its value (mixed over
    the heads); one step further back it is gone."""
    from tinyserve_b200.kernels import ops

    heads, groups, total = 4, 2, 400
    talk = torch.eye(heads, device="cuda") * 0.5 + 0.25
    for window in (1, 2, page - 1, page, page + 1, 5 * page, 133, 300):
        for back in {0, 1, window - 1, window, window + 1, min(window, 2 * page), total - 1}:
            far = total - 1 - back
            if far < 0:
                continue
            tables, table, pages = _tables([total, 9], page, 3)
            k, v = _stores(dtype, tables, pages, page, [total, 9], groups, d, d)
            k = k * 0.05
            where = tables[0][far // page], far % page
            k[where[0], :, where[1]] = 4.0
            q = _rand(new + 1, heads, d, seed=3, scale=0.05, dtype=dtype)
            q[new - 1] = 4.0
            res = []
            for impl in (ops, refs):
                out = torch.empty(new + 1, heads * d, dtype=dtype, device="cuda")
                ctx = Ctx([new, 1], [total, 9])
                if mixer == "mixed":
                    impl.talking_attention(q, k, v, page, table, ctx, d ** -0.5, window, 60.0, talk, out)
                else:
                    impl.paged_attention(q, k, v, page, table, ctx, d ** -0.5, window, out, sinks=torch.full((heads,), -20.0, device="cuda"))
                res.append(out.float())
            torch.testing.assert_close(res[0], res[1], atol=3e-2 if dtype == torch.bfloat16 else 3e-5, rtol=2e-2 if dtype == torch.bfloat16 else 3e-5)
            value = v[where[0], :, where[1]].float().repeat_interleave(heads // groups, 0)
            factor = talk.sum(1)[:, None] if mixer == "mixed" else 1.0
            got = res[0][new - 1].view(heads, d)
            if back < window:
                torch.testing.assert_close(got, factor * value, atol=3e-2, rtol=2e-2)
            elif window > 1:
                assert (got - factor * value).abs().max() > 0.3, (window, back)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, groups, d, dv, rotary, interleaved, unit", [(4, 2, 32, 32, 16, True, True), (3, 1, 64, 64, 64, True, False), (2, 2, 128, 64, 32, False, True),
                                                                             (5, 5, 12, 20, 6, True, True), (1, 1, 17, 9, 0, True, False), (6, 2, 48, 48, 48, True, True),
                                                                             (2, 1, 24, 24, 10, False, True)])
def test_convolution_rotation_and_unit_norm_kernel(dtype, heads, groups, d, dv, rotary, interleaved, unit) -> None:
    """Portions of several lengths (also shorter than the taps) and single tokens, from and to state slots out of order;
    the rows are the first columns of a wider matrix. Foreign slots and pages stay as they are."""
    from tinyserve_b200.kernels import ops

    page, channels = 4, (heads + groups) * d + groups * dv
    for taps in (None, 1, 2, 4, 6):
        for lens in ([5, 1, 2, 33, 3], [1, 1, 1]):
            t = sum(lens)
            proj = _rand(t, channels + 8, seed=1, dtype=dtype)
            w = None if taps is None else _rand(taps, channels, seed=2, scale=0.5, dtype=dtype)
            cos = sin = None
            if rotary:
                ang = (torch.arange(t, dtype=torch.float64)[:, None] * 7 % 900) * (1e3 ** (-torch.arange(0, rotary, 2, dtype=torch.float64) / rotary))[None, :]
                cos, sin = (ang.cos() * 1.1).float().cuda(), (ang.sin() * 1.1).float().cuda()
            slots = torch.randperm(16 * page, generator=torch.Generator().manual_seed(4))[:t].int().cuda()
            rows = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(5))[: len(lens)].tolist()
            start = _rand(len(lens) + 3, max(1, (taps or 1) - 1) * channels, seed=6)
            res = []
            for impl in (ops, refs):
                ctx = FakeStep(lens, rows, device="cuda")
                state = start.clone()
                kc = torch.full((16, groups, page, d), float("nan"), dtype=dtype, device="cuda")
                vc = torch.full((16, groups, page, dv), float("nan"), dtype=dtype, device="cuda")
                qo = torch.empty(t, heads, d, dtype=dtype, device="cuda")
                impl.qkv_rotate(proj, w, state if taps is not None and taps > 1 else None, ctx, cos, sin, rotary, interleaved, 1e-6 if unit else None,
                                slots, kc, vc, page, heads, groups, d, dv, qo)
                res.append((qo.float(), kc.float(), vc.float(), state))
            for got, want in zip(*res):
                torch.testing.assert_close(got, want, equal_nan=True, **_tol(dtype))
            untouched = [s for s in range(len(lens) + 3) if s not in rows]
            assert torch.equal(res[0][3][untouched], start[untouched])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, dv, rotary, interleaved", [(2, 16, 24, 16, False), (1, 40, 16, 8, False), (3, 8, 8, 2, True), (2, 64, 64, 64, False), (1, 128, 40, 64, True),
                                                               (1, 256, 32, 256, False), (2, 20, 12, 0, False)])
def test_retention_kernel(dtype, heads, d, dv, rotary, interleaved) -> None:
    """Prompt portions, single tokens and a portion long enough to run in segments, from and to state slots out of
    order; decays of one, near one and small; q, k, v are column slices of one product."""
    from tinyserve_b200.kernels import ops

    decay = torch.tensor([1.0, 0.995, 0.6][:heads], device="cuda")
    for lens in ([5, 1, 33, 1, 2], [1, 1, 1], [300, 7, 1], [16, 17]):
        t = sum(lens)
        wide = _rand(t, 2 * heads * d + heads * dv + 3, seed=1, scale=0.5, dtype=dtype)
        q, k, v = wide[:, : heads * d], wide[:, heads * d: 2 * heads * d], wide[:, 2 * heads * d: 2 * heads * d + heads * dv]
        cos = sin = None
        if rotary:
            ang = torch.arange(t, dtype=torch.float64)[:, None] * (1e4 ** (-torch.arange(0, rotary, 2, dtype=torch.float64) / rotary))[None, :]
            cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
        slots = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(5))[: len(lens)].tolist()
        start = _rand(len(lens) + 3, heads * d * dv, seed=4, scale=0.3)
        res = []
        for impl in (ops, refs):
            state = start.clone()
            ctx = FakeStep(lens, slots, device="cuda")
            ctx.arena = Arena()
            out = torch.full((t, heads, dv), float("nan"), device="cuda")
            impl.linear_scan_rotated(q, k, v, decay, cos, sin, rotary, interleaved, d ** -0.5, state, ctx, heads, d, dv, out)
            res.append((out, state))
        tol = 3e-5 * max(1.0, float(res[1][0].abs().max()))        # nothing behind the projections is rounded, in either mode
        torch.testing.assert_close(res[0][0], res[1][0], atol=tol, rtol=tol)
        torch.testing.assert_close(res[0][1], res[1][1], atol=tol, rtol=tol)
        untouched = [s for s in range(len(lens) + 3) if s not in slots]
        assert torch.equal(res[0][1][untouched], start[untouched])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, experts, top, hidden, ff", [(1, 1, 1, 64, 24), (9, 4, 2, 64, 24), (64, 5, 5, 72, 40), (300, 6, 1, 128, 64), (700, 8, 3, 256, 256),
                                                              (1500, 16, 4, 512, 256)])
def test_experts_with_weights_on_their_input_from_routing_to_combine(dtype, tokens, experts, top, hidden, ff) -> None:
    """Sigmoid scores that are not normalised and multiply the experts' input, and the clamped activation, at sizes
    that take each form of the experts' products; sums beyond both limits occur."""
    from tinyserve_b200.kernels import ops

    x, limit = _rand(tokens, hidden, seed=1, dtype=dtype), 0.9
    w_router = _rand(experts, hidden, seed=2, scale=0.2, dtype=dtype)
    w_gu, w_down = _rand(experts, 2 * ff, hidden, seed=3, scale=0.15, dtype=dtype), _rand(experts, hidden, ff, seed=4, scale=0.1, dtype=dtype)
    rule = ops.RouteRule(scored=True, sigmoid=True, normalise=False, on_input=True)
    res = []
    for impl in (ops, refs):
        arena, counts = Arena(), torch.zeros(experts, dtype=torch.int32, device="cuda")
        tile_rows = impl.moe_tile_rows(tokens, top, experts, dtype, (hidden, ff))
        plan = impl.moe_route_from(x, w_router, top, counts, arena, tile_rows, rule, experts)
        act = torch.full((tokens * top, ff), float("nan"), dtype=dtype, device="cuda")
        impl.moe_gemm(x, w_gu, act, plan, gated=True, gather=True, arena=arena, limit=limit)
        y = torch.full((tokens * top, hidden), float("nan"), dtype=dtype, device="cuda")
        impl.moe_gemm(act, w_down, y, plan, gated=False, gather=False, arena=arena)
        out = torch.empty(tokens, hidden, dtype=dtype, device="cuda")
        impl.moe_combine(y, plan, None, out)
        assert int(counts.abs().sum()) == 0
        res.append((out.float(), plan))
    (got, plan), (want, ref_plan) = res
    rows = plan["row_of"].long()
    assert torch.equal(plan["row_weight"][rows], plan["weights"])
    if dtype == torch.float32:
        assert torch.equal(plan["ids"], ref_plan["ids"])
        torch.testing.assert_close(plan["weights"], ref_plan["weights"], atol=1e-6, rtol=1e-5)
        torch.testing.assert_close(got, want, atol=2e-4, rtol=2e-4)
    else:
        same = (plan["ids"].view(tokens, top) == ref_plan["ids"].view(tokens, top)).all(-1)      # rounding may flip a close call
        assert float(same.float().mean()) > 0.97
        torch.testing.assert_close(got[same], want[same], atol=2e-2 * float(want.abs().max()), rtol=6e-2)


@pytest.mark.parametrize("tokens", [3, 65])
def test_sigmoid_scores_near_one_are_told_apart(tokens) -> None:
    """Logits so large that their sigmoids round to the same value: the largest logit is picked all the same."""
    from tinyserve_b200.kernels import ops

    logits = 30.0 + torch.arange(12.0).flip(0).repeat(tokens, 1).roll(3, 1).cuda()
    rule = ops.RouteRule(scored=True, sigmoid=True, normalise=False, on_input=True)
    plan = ops.moe_route(logits, 2, torch.zeros(12, dtype=torch.int32, device="cuda"), Arena(), rule=rule)
    assert plan["ids"].view(tokens, 2).tolist() == [[3, 4]] * tokens


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, hidden", [(1, 48), (37, 256), (5, 37), (300, 1024)])
def test_norm_that_folds_two_outputs_and_a_pass_vector_kernel(dtype, rows, hidden) -> None:
    from tinyserve_b200.kernels import ops

    x, first = _rand(rows, hidden, seed=1, scale=2.0), _rand(rows, hidden, seed=2)
    a, b = _rand(rows, hidden, seed=3, dtype=dtype), _rand(rows, hidden, seed=4, dtype=dtype)
    table, w = _rand(3, hidden, seed=5, dtype=dtype), _rand(hidden, seed=6, scale=0.3, dtype=dtype)
    pick = torch.tensor([rows - 1, 0], dtype=torch.int32, device="cuda")
    for add_rows, add_vec, with_b, with_a in ((None, table[1], False, False), (first, table[2], False, True), (None, None, True, True), (first, table[0], True, True)):
        for chosen in (None, pick):
            res = []
            for impl in (ops, refs):
                xs = x.clone()
                out = torch.empty(rows if chosen is None else 2, hidden, dtype=dtype, device="cuda")
                impl.post_norm_add_rms_norm(xs, a if with_a else None, None, None, 0.0, False, w, True, 1e-6, out, rows=chosen, post_mult=0.6,
                                            second=b if with_b else None, second_scale=1.7, add_rows=add_rows, add_vec=add_vec)
                res.append((xs, out.float()))
            torch.testing.assert_close(res[0][0], res[1][0], atol=1e-5, rtol=1e-5)
            torch.testing.assert_close(res[0][1], res[1][1], **_tol(dtype))
            assert chosen is None or torch.equal(res[0][0], x)


# ------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {k: write_model(tmp_path_factory.mktemp("sanevik" + k), k) for k in CONFIGS}


LENGTHS = {"A": [1, 2, 9, 37, 70, 131], "B": [3, 33, 64, 97], "C": [5, 18, 40, 100], "D": [2, 47, 160]}


@pytest.fixture(scope="module")
def oracle(folders):
    out = {}
    for which in CONFIGS:
        vocab = plain.read_config(folders[which])["vocab"]
        reqs = {f"r{i}": random_prompt(n, vocab, 200 + 7 * i) for i, n in enumerate(LENGTHS[which])}
        out[which] = (reqs, {rid: plain_oracle(folders[which], toks) for rid, toks in reqs.items()})
    return out


def _check(got, reqs, want, dtype, what) -> None:
    assert all(sorted(got[rid]) == list(range(len(reqs[rid]))) for rid in got)
    rows = torch.cat([torch.stack([got[rid][p] for p in range(len(reqs[rid]))]) for rid in got])
    assert_rows_close(rows, torch.cat([want[rid][0] for rid in got]), torch.cat([want[rid][1] for rid in got]), dtype, what)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which, page", [("A", 4), ("A", 16), ("B", 8), ("B", 16), ("C", 16), ("C", 32), ("D", 16), ("D", 8)])
def test_model_under_every_cut(folders, oracle, dtype, which, page) -> None:
    """Whole prompts, token by token at the end, portions down to two tokens, and mixed batches, with NaN in the pages
    and slots that no request owns."""
    from tinyserve_b200.model import DecoderModel

    reqs, want = oracle[which]
    model = DecoderModel.from_folder(folders[which], dtype, "cuda")
    plans = [cases.mixed(reqs, 3), cases.mixed(reqs, 4, max_live=2)]
    for rid, toks in reqs.items():
        plans += [cases.whole(rid, toks), cases.tail_decoded(rid, toks, 32), cases.portions(rid, toks, 1)]
    for n, steps in enumerate(plans):
        got, _ = run_steps(model, page, steps, cases.max_live_tokens(steps))
        _check(got, reqs, want, dtype, f"{which}, schedule {n}")


@pytest.mark.parametrize("seed", list(range(1, 11)))
def test_configurations_drawn_at_random(seed, tmp_path) -> None:
    from tinyserve_b200.model import DecoderModel

    cfg = random_config(seed)
    folder = write_model(tmp_path, cfg, seed)
    reqs = {f"r{i}": random_prompt(n, cfg["vocab"], 300 + seed + 7 * i) for i, n in enumerate([2, 35, 80, 61])}
    want = {rid: plain_oracle(folder, toks) for rid, toks in reqs.items()}
    page = [4, 8, 16, 32][seed % 4]
    plans = [cases.mixed(reqs, seed), cases.whole("r2", reqs["r2"]), cases.tail_decoded("r2", reqs["r2"], 40), cases.portions("r3", reqs["r3"], seed)]
    for dtype in DTYPES:
        model = DecoderModel.from_folder(folder, dtype, "cuda")
        for n, steps in enumerate(plans):
            got, _ = run_steps(model, page, steps, cases.max_live_tokens(steps))
            _check(got, reqs, want, dtype, f"seed {seed}, schedule {n}: {json.dumps(cfg)[:300]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts(dtype, tmp_path) -> None:
    """A prompt of several hundred tokens at the sizes of the tensor-core kernels: the retention of a long portion runs
    in segments, windows pass over prompt and decoded tokens, a decoded token's keys are cut into ranges."""
    from tinyserve_b200.kernels import ops
    from tinyserve_b200.model import DecoderModel

    folder = write_model(tmp_path, CONFIG_D, 31)
    vocab = CONFIG_D["vocab"]
    reqs = {"long": random_prompt(420, vocab, 41), "short": random_prompt(9, vocab, 43)}
    assert ops.linear_scan_segments(420, 1, 2, 64, 64)[1] > 1
    want = {rid: plain_oracle(folder, toks) for rid, toks in reqs.items()}
    model = DecoderModel.from_folder(folder, dtype, "cuda")
    plans = [cases.whole("long", reqs["long"]), cases.tail_decoded("long", reqs["long"], 20),
             cases.portions("long", reqs["long"], 1, sizes=(300, 257, 2, 100)), cases.mixed(reqs, 2)]
    for n, steps in enumerate(plans):
        got, _ = run_steps(model, 16, steps, cases.max_live_tokens(steps))
        _check(got, {rid: reqs[rid] for rid in got}, want, dtype, f"long prompts, schedule {n}")


def test_batch_mates_pages_and_slots_do_not_matter(folders, oracle) -> None:
    """float32: a request's logits alone, beside others, and again on the pages and in the slot that another request has
    just given back, agree to rounding."""
    from tinyserve_b200.engine.replay import Replayer
    from tinyserve_b200.model import DecoderModel

    reqs, _ = oracle["A"]
    model = DecoderModel.from_folder(folders["A"], torch.float32, "cuda")
    toks, other = reqs["r4"], reqs["r5"]
    rep = Replayer(model, 256, page_size=4, max_live=2)
    alone = rep.run_step([("x", toks, [len(toks) - 1])], ["x"]).clone()
    rep.run_step([("y", other[:50], [])], [])
    beside = rep.run_step([("y", other[50:51], []), ("x", toks, [len(toks) - 1])], ["x", "y"]).clone()
    rep.run_step([("z", toks[:7], []), ("w", other[:3], [])], [])
    again = rep.run_step([("w", other[3:4], []), ("z", toks[7:], [len(toks) - 8])], ["z", "w"]).clone()
    torch.testing.assert_close(beside, alone, atol=2e-5, rtol=2e-5)
    torch.testing.assert_close(again, alone, atol=2e-5, rtol=2e-5)
    assert rep.cache.state_pool.num_free == 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "D"])
def test_long_decoding(folders, dtype, which) -> None:
    from tinyserve_b200.model import DecoderModel

    vocab = plain.read_config(folders[which])["vocab"]
    toks = random_prompt(130, vocab, 9)
    want = plain_oracle(folders[which], toks)
    model = DecoderModel.from_folder(folders[which], dtype, "cuda")
    got, _ = run_steps(model, 16, cases.tail_decoded("a", toks, 125), 192)
    assert_rows_close(torch.stack([got["a"][p] for p in range(130)]), *want, dtype, "all tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "D"])
def test_overlapping_launches_change_no_bit(folders, oracle, dtype, which) -> None:
    """A kernel that starts while the kernels before it still run must read their results behind its wait: the logits
    of mixed steps, decoded tokens and portions are equal bit for bit with the overlap on and off."""
    from test_diderax_gpu import _with_overlap
    from tinyserve_b200.model import DecoderModel

    reqs, _ = oracle[which]
    model = DecoderModel.from_folder(folders[which], dtype, "cuda")
    long = list(reqs)[-1]
    for steps in (cases.mixed(reqs, 5), cases.tail_decoded(long, reqs[long], 40), cases.portions(long, reqs[long], 3)):
        rows = {}
        for mask in (0, -1):
            got, _ = _with_overlap(mask, lambda: run_steps(model, 16, steps, cases.max_live_tokens(steps)))
            rows[mask] = torch.cat([torch.stack([got[r][p] for p in sorted(got[r])]) for r in sorted(got)])
        assert torch.equal(rows[0], rows[-1])


def test_a_long_prompt_at_a_real_width_with_overlapping_launches() -> None:
    """2,048 tokens at width 1,024 through both layer kinds and a loop, experts in tiles of 128 sorted rows: two
    different prompts one after the other on the same scratch, overlap on and off, equal bit for bit."""
    from test_diderax_gpu import _with_overlap
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.engine.replay import Replayer
    from tinyserve_b200.model import DecoderModel

    mlp = {"kind": "moe", "router": {"experts": 16, "top": 3}, "expert": {"ff": 512, "limit": 5.0}}
    attn = {"heads": 16, "kv_heads": 8, "dim": 64, "vdim": 64, "scale": 0.1, "rot": {"dims": 32, "base": 1e4}, "mask": {"size": 300}}
    right = {"heads": 8, "dim": 64, "vdim": 64, "rot": {"dims": 64, "base": 1e4}, "decay": [0.99] * 8}
    cfg = {"architecture": "Sanevik", "vocab": 1000, "width": 1024, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 2}, "layers": [
        {"type": "attention", "mixer": attn, "mlp": mlp},
        {"type": "parallel", "mixer": {"left": {**attn, "softcap": 20.0, "conv": 4}, "right": right, "left_scale": 0.5, "right_scale": 0.5}, "mlp": mlp}]}
    model = DecoderModel.from_config(config_from_dict(cfg), seed=1, dtype=torch.bfloat16, device="cuda")
    prompts = [random_prompt(2048, 1000, s) for s in (1, 2)]

    def run():
        rep = Replayer(model, 4096, page_size=16, max_live=2)
        return torch.cat([rep.run_step([(f"p{i}", p, [0, 1000, 2047])], [f"p{i}"]).clone() for i, p in enumerate(prompts)])

    plain_rows, overlapped = _with_overlap(0, run), _with_overlap(-1, run)
    assert not plain_rows.isnan().any() and torch.equal(plain_rows, overlapped)


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("which", ["A", "B", "D"])
def test_greedy_generation_through_llm(folders, graphs, which) -> None:
    from tinyserve_b200 import LLM

    cfg, w = plain.read_config(folders[which]), plain.read_weights(folders[which], torch.float64)
    prompts = [random_prompt(n, cfg["vocab"], 40 + n) for n in (3, 11, 26)]
    want = [plain.greedy(cfg, w, p, 6) for p in prompts]
    llm = LLM.from_folder(folders[which], dtype="float32", page_size=8, num_pages=64, max_num_seqs=2, max_batch_tokens=16,
                          chunked_prefill=True, decode_graphs=graphs)
    assert llm.generate(prompts, max_new_tokens=6) == want
    assert (llm.engine.runner.num_graph_steps > 0) == graphs
    assert all(g.allocator.num_used == 0 for g in llm.cache.groups)


def test_command_line(folders) -> None:
    cfg, w = plain.read_config(folders["A"]), plain.read_weights(folders["A"], torch.float64)
    prompt = random_prompt(19, cfg["vocab"], 77)
    want = plain.greedy(cfg, w, prompt, 8)
    cmd = [sys.executable, str(ROOT / "bin" / "generate"), "--model-dir", str(folders["A"]), "--prompt-ids", ",".join(map(str, prompt)),
           "--max-new-tokens", "8", "--dtype", "float32", "--block-size", "8"]
    out = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert f"new ids:    {want}" in out.stdout


def test_trace_run_subprocess(folders, oracle, tmp_path) -> None:
    reqs, want = oracle["C"]
    steps = cases.mixed(reqs, 6, max_live=3)
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": p} for r, t, p in entries], "end": end})
             for i, (entries, end) in enumerate(steps)]
    out = tmp_path / "out"
    vocab = plain.read_config(folders["C"])["vocab"]
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folders["C"]), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", str(cases.max_live_tokens(steps)), "--max-requests", "3"],
                          input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [x for x in proc.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    fed: dict[str, int] = {}
    for i, (entries, _) in enumerate(steps):
        wanted = sum(len(p) for _, _, p in entries)
        rows = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, vocab)) if wanted else None
        at = 0
        for rid, toks, places in entries:
            base = fed.get(rid, 0)
            for p in places:
                w, c = want[rid]
                assert_rows_close(rows[at][None], w[base + p][None], c[base + p][None], torch.float32, f"{rid} at {base + p}")
                at += 1
            fed[rid] = base + len(toks)
