"""Risonex on the GPU: every new kernel form alone against its reference at sizes other than any model's, with
inputs made so that a fault shows (a key that carries all the weight just inside and just outside a chunk, at page
borders and far back; NaN in pages and slots that belong to nobody); the whole model in float32 and bfloat16
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
import plain_risonex as plain
import replay_cases as cases
from fegilix_cases import FakeStep, run_steps
from risonex_cases import CONFIGS, CONFIG_D, assert_rows_close, oracle as plain_oracle, random_config, write_model
from test_diderax_gpu import DTYPES, ROOT, Arena, Ctx, _rand, _tables, _tol, _with_overlap
from test_sanevik_gpu import _stores
from tiny_configs import random_prompt

pytestmark = pytest.mark.gpu


def _both(impl, q, k, v, page, table, ctx, scale, chunk, factor, mult, window=0):
    """The finished heads of differential attention; the scratch starts as NaN."""
    t, heads, _ = q.shape
    dv = v.shape[3]
    maps = torch.full((t, heads * 2 * dv), float("nan"), dtype=q.dtype, device="cuda")
    out = torch.full((t, heads * dv), float("nan"), dtype=q.dtype, device="cuda")
    impl.paged_attention(q, k, v, page, table, ctx, scale, window, maps, chunk=chunk, maps=2, finish=(out, factor, mult, 1e-6))
    return out.float().view(t, heads, dv)


# ------------------------------------------------------------ kernels one by one
SIZES = [(4, 2, 64, 128, 16), (2, 2, 64, 128, 8), (6, 1, 64, 128, 32), (4, 4, 32, 64, 16), (20, 2, 32, 64, 8), (4, 2, 24, 48, 16), (3, 1, 56, 112, 4),
         (2, 1, 128, 256, 16), (5, 5, 12, 20, 4), (4, 2, 200, 72, 8), (1, 1, 16, 32, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, groups, d, dv, page", SIZES)
@pytest.mark.parametrize("chunk, window", [(0, 0), (37, 0), (1, 0), (64, 0), (130, 0), (256, 0), (0, 50)])
def test_differential_attention_kernels(dtype, heads, groups, d, dv, page, chunk, window) -> None:
    """Prompt portions beside single tokens, portions alone, and steps of single tokens alone (their keys are cut into
    ranges), at sizes that take each of the kernels: finished inside the tcgen05 kernel, mma.sync and CUDA cores."""
    factor = torch.tensor([0.7], device="cuda")
    for lens, news in (([page * 3 + 1, 170, 33, 1, 300], [1, 17, 33, 1, 90]), ([300, 64, 129], [260, 64, 129]), ([600, 350, 513, 1], [1, 1, 1, 1])):
        tables, table, pages = _tables(lens, page, 7)
        k, v = _stores(dtype, tables, pages, page, lens, groups, 2 * d, dv)
        q = _rand(sum(news), heads, 2 * d, seed=3, dtype=dtype)
        got, want = (_both(impl, q, k, v, page, table, Ctx(news, lens), d ** -0.5, chunk, factor, 0.8, window) for impl in (_ops(), refs))
        assert not got.isnan().any()
        tol = 5e-5 if dtype == torch.float32 else 4e-2      # each map is rounded to bfloat16 before they are combined, where they are
        loose = (got - want).abs() > tol * max(1.0, float(want.abs().max()))
        # a row whose maps nearly cancel is divided by a small root mean square: bfloat16 loses the digits that cancelled
        assert float(loose.float().mean()) <= (0.0 if dtype == torch.float32 else 2e-3), float(loose.float().mean())


def _ops():
    from tinyserve_b200.kernels import ops

    return ops


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, groups, d, page", [(4, 2, 64, 16), (2, 1, 128, 8), (8, 2, 128, 16), (4, 4, 48, 4), (3, 1, 80, 16)])
@pytest.mark.parametrize("prefill", ["tcgen05", "mma"])
def test_chunks_with_one_map(dtype, heads, groups, d, page, prefill) -> None:
    """The mask of chunks in the kernels of ordinary heads, also in the prompt kernel that is not the default."""
    ops = _ops()
    saved, ops.PREFILL_ATTENTION = ops.PREFILL_ATTENTION, prefill
    try:
        for chunk in (1, 16, 37, 128, 200):
            for lens, news in (([page * 3 + 1, 170, 33, 1, 300], [1, 17, 33, 1, 290]), ([600, 350, 513, 1], [1, 1, 1, 1])):
                tables, table, pages = _tables(lens, page, 7)
                k, v = _stores(dtype, tables, pages, page, lens, groups, d, d)
                q = _rand(sum(news), heads, d, seed=3, dtype=dtype)
                res = []
                for impl in (ops, refs):
                    out = torch.full((sum(news), heads * d), float("nan"), dtype=dtype, device="cuda")
                    impl.paged_attention(q, k, v, page, table, Ctx(news, lens), d ** -0.5, 0, out, chunk=chunk)
                    res.append(out.float())
                torch.testing.assert_close(res[0], res[1], **_tol(dtype))
    finally:
        ops.PREFILL_ATTENTION = saved


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("new", [1, 2, 70, 150])
@pytest.mark.parametrize("d, dv, page", [(64, 128, 16), (32, 64, 8), (20, 24, 4)])
def test_a_key_just_inside_and_just_outside_the_chunk(dtype, new, d, dv, page) -> None:
    """One key outweighs all others for one map of the last query. While it lies in the query's chunk the map gives its
    value; one position before the chunk's start it is gone. The other map sees ordinary scores."""
    heads, groups, factor = 4, 2, torch.tensor([0.5], device="cuda")
    for total in (257, 400, 512):
        for chunk in (1, 2, page - 1, page, page + 1, 100, 128, 133, 300):
            first = (total - 1) // chunk * chunk
            for far in {first, first - 1, first - chunk, min(total - 1, first + 1), total - 1, (total - 1) // page * page, 0}:
                if not 0 <= far < total or (far < first and first - far > 2 * chunk and far):
                    continue
                tables, table, pages = _tables([total, 9], page, 3)
                k, v = _stores(dtype, tables, pages, page, [total, 9], groups, 2 * d, dv)
                k = k * 0.05
                where = tables[0][far // page], far % page
                k[where[0], :, where[1], d:] = 4.0
                q = _rand(new + 1, heads, 2 * d, seed=3, scale=0.05, dtype=dtype)
                q[new - 1, :, d:] = 4.0
                got, want = (_both(impl, q, k, v, page, table, Ctx([new, 1], [total, 9]), d ** -0.5, chunk, factor, 1.0) for impl in (_ops(), refs))
                torch.testing.assert_close(got[new - 1], want[new - 1], atol=6e-2 if dtype == torch.bfloat16 else 5e-5, rtol=5e-2 if dtype == torch.bfloat16 else 5e-5)
                # the map that points at the far key, alone
                value = v[where[0], :, where[1]].float().repeat_interleave(heads // groups, 0)
                alone, _ = (_both(impl, q, k, v, page, table, Ctx([new, 1], [total, 9]), d ** -0.5, chunk, torch.tensor([1e4], device="cuda"), 1.0)
                            for impl in (_ops(), refs))
                unit = value / value.pow(2).mean(-1, keepdim=True).sqrt()
                if far >= first:
                    torch.testing.assert_close(-alone[new - 1], unit, atol=4e-2, rtol=2e-2)
                elif chunk > 1:
                    assert (-alone[new - 1] - unit).abs().max() > 0.3, (chunk, far)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dv", [(1, 8), (4, 128), (3, 256), (5, 37)])
def test_combination_of_two_maps_kernel(dtype, heads, dv) -> None:
    """All rows, and only the rows of listed requests (the others keep what they hold)."""
    ops = _ops()
    x, factor = _rand(9, heads * 2 * dv, seed=1, dtype=dtype), torch.tensor([-1.3], device="cuda")
    ctx = Ctx([1, 4, 1, 3], [5, 9, 1, 3])
    for rows_of in (None, (ctx.decode_seqs, ctx)):
        res = []
        for impl in (ops, refs):
            out = torch.full((9, heads * dv), 7.0, dtype=dtype, device="cuda")
            impl.pair_combine(x, factor, 1e-5, 0.6, out, heads, dv, rows_of=rows_of)
            res.append(out.float())
        torch.testing.assert_close(res[0], res[1], **_tol(dtype))
        assert rows_of is None or (bool((res[0][1:5] == 7.0).all()) and bool((res[0][6:] == 7.0).all()) and not bool((res[0][[0, 5]] == 7.0).any()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, groups, d, dv, rotary", [(4, 2, 32, 64, 0), (3, 1, 12, 20, 0), (2, 2, 64, 128, 16), (5, 5, 7, 9, 0), (1, 1, 128, 256, 0)])
def test_keys_of_two_maps_side_by_side(dtype, heads, groups, d, dv, rotary) -> None:
    ops = _ops()
    t, page = 21, 4
    q_rows, k_rows, v_rows = heads * 2 * d, groups * 2 * d, groups * dv
    wide = _rand(t, q_rows + k_rows + v_rows, seed=1, scale=2.0, dtype=dtype)
    qw, kw = (1 + _rand(d, seed=2, scale=0.3)).to(dtype), (1 + _rand(d, seed=3, scale=0.3)).to(dtype)
    cos = sin = None
    if rotary:
        ang = torch.arange(50, 50 + t, dtype=torch.float64)[:, None] * (1e3 ** (-torch.arange(0, rotary, 2, dtype=torch.float64) / rotary))[None, :]
        cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
    slots = torch.randperm(8 * page, generator=torch.Generator().manual_seed(4))[:t].int().cuda()
    res = []
    for impl in (ops, refs):
        kc = torch.full((8, groups, page, 2 * d), float("nan"), dtype=dtype, device="cuda")
        vc = torch.full((8, groups, page, dv), float("nan"), dtype=dtype, device="cuda")
        qo = torch.empty(t, heads * 2, d, dtype=dtype, device="cuda")
        impl.qkv_prepare(wide[:, :q_rows], wide[:, q_rows: q_rows + k_rows], wide[:, q_rows + k_rows:], qw, kw, 1e-6, cos, sin, rotary, slots, kc, vc, page,
                         heads * 2, groups, d, dv, qo, maps=2)
        res.append((qo.float(), kc.float(), vc.float()))
    for got, want in zip(*res):
        torch.testing.assert_close(got, want, equal_nan=True, **_tol(dtype))


@pytest.mark.parametrize("chunks", [True, False])
@pytest.mark.parametrize("heads, groups, d, dv", [(2, 1, 16, 24), (4, 2, 40, 16), (3, 3, 8, 8), (4, 1, 64, 64), (2, 2, 128, 40), (1, 1, 256, 32), (6, 2, 20, 12),
                                                  (24, 2, 128, 64), (5, 1, 50, 130), (3, 1, 7, 67)])
def test_state_space_scan_kernel(heads, groups, d, dv, chunks, monkeypatch) -> None:
    """Prompt portions, single tokens and portions long enough to run in segments, from and to state slots out of order;
    rates from slow to fast, step sizes over several orders of magnitude; C, B and x are column slices. Long portions as
    products over chunks of tokens and, with that switched off (and where the state is too wide), token by token."""
    ops = _ops()
    monkeypatch.setattr(ops, "STATE_SPACE_CHUNKS", chunks)
    a_log, skip = torch.linspace(-4.0, 2.0, heads, device="cuda"), _rand(heads, seed=7)
    bias = torch.linspace(-3.0, 1.0, heads, device="cuda")
    for lens in ([5, 1, 33, 1, 2], [1, 1, 1], [300, 7, 1], [16, 17], [700, 260], [1, 1, 128, 1, 65, 64, 2], [63, 193]):
        t = sum(lens)
        wide = _rand(t, 2 * groups * d + heads * dv + 3, seed=1, scale=0.5)
        x, b, c = wide[:, : heads * dv], wide[:, heads * dv: heads * dv + groups * d], wide[:, heads * dv + groups * d: heads * dv + 2 * groups * d]
        step = _rand(t, heads + 5, seed=2, scale=2.0)[:, :heads]
        slots = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(5))[: len(lens)].tolist()
        start = _rand(len(lens) + 3, heads * d * dv, seed=4, scale=0.3)
        res = []
        for impl, up in ((ops, torch.float32), (refs, torch.float64)):
            state = start.clone().to(up)
            ctx = FakeStep(lens, slots, device="cuda")
            ctx.arena = Arena()
            out = torch.full((t, heads, dv), float("nan"), dtype=up, device="cuda")
            impl.state_space_scan(c, b, x, step, bias, a_log, skip, state, ctx, heads, groups, d, dv, out)
            res.append((out.double(), state.double()))
        tol = 3e-5 * max(1.0, float(res[1][0].abs().max()))
        torch.testing.assert_close(res[0][0], res[1][0], atol=tol, rtol=tol)
        torch.testing.assert_close(res[0][1], res[1][1], atol=tol, rtol=tol)
        untouched = [s for s in range(len(lens) + 3) if s not in slots]
        assert torch.equal(res[0][1][untouched], start[untouched].double())


@pytest.mark.parametrize("chunks", [True, False])
def test_a_state_a_thousand_tokens_old_is_still_read(chunks, monkeypatch) -> None:
    """One write that decays slowly, then steps that write next to nothing: the read-out far behind it is its value."""
    ops = _ops()
    monkeypatch.setattr(ops, "STATE_SPACE_CHUNKS", chunks)
    heads, d, dv, t = 2, 16, 8, 1200
    x, b, c = torch.zeros(t, heads * dv, device="cuda"), torch.zeros(t, heads * d, device="cuda"), torch.zeros(t, heads * d, device="cuda")
    x[0], b[0], c[-1] = 3.0, 1.0, 1.0
    step = torch.full((t, heads), -12.0, device="cuda")
    step[0] = 4.0
    a_log = torch.full((heads,), -2.0, device="cuda")
    zero = torch.zeros(heads, device="cuda")
    for cuts in ([t], [1, t - 1], [600, 300, 299, 1], [t - 1, 1]):
        state = torch.zeros(2, heads * d * dv, device="cuda")
        at = 0
        for n in cuts:
            ctx = FakeStep([n], [1], device="cuda")
            ctx.arena = Arena()
            out = torch.empty(n, heads, dv, device="cuda")
            s = slice(at, at + n)
            ops.state_space_scan(c[s], b[s], x[s], step[s], zero, a_log, zero, state, ctx, heads, heads, d, dv, out)
            at += n
        dt0, later = np.log1p(np.exp(4.0)), np.log1p(np.exp(-12.0)) * (t - 1)
        want = dt0 * 3.0 * d * np.exp(-np.exp(-2.0) * later)
        torch.testing.assert_close(out[-1], torch.full((heads, dv), float(want), device="cuda"), rtol=1e-4, atol=0.0)


def test_a_weak_decay_behind_a_strong_one_keeps_its_digits() -> None:
    """Within a chunk one token decays everything before it to nothing; what is written behind it decays by very little. The
    differences of large running sums still give those small decays to 32-bit accuracy."""
    ops = _ops()
    heads, d, dv, t = 2, 24, 16, 192
    x, b, c = _rand(t, heads * dv, seed=1), _rand(t, heads * d, seed=2), _rand(t, heads * d, seed=3)
    step = torch.full((t, heads), -6.0, device="cuda")
    step[5::40] = 9.0
    a_log = torch.tensor([6.0, 3.0], device="cuda")
    zero = torch.zeros(heads, device="cuda")
    res = []
    for impl, up in ((ops, torch.float32), (refs, torch.float64)):
        state = torch.zeros(2, heads * d * dv, dtype=up, device="cuda")
        ctx = FakeStep([t], [1], device="cuda")
        ctx.arena = Arena()
        out = torch.empty(t, heads, dv, dtype=up, device="cuda")
        impl.state_space_scan(c, b, x, step, zero, a_log, zero, state, ctx, heads, heads, d, dv, out)
        res.append(out.double())
    quiet = torch.ones(t, dtype=torch.bool)
    for n in range(5, t, 40):
        quiet[n: n + 3] = False               # right behind the strong token its own large write dominates
    scale = res[1][quiet].abs().median()
    assert float((res[0] - res[1])[quiet].abs().max()) < 2e-5 * max(1.0, float(res[1].abs().max())) and float(scale) > 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 8])
def test_convolution_with_a_bias_kernel(dtype, taps) -> None:
    """Portions of several lengths (also shorter than the taps), and a step of single tokens (one kernel then)."""
    ops = _ops()
    channels = 300
    for lens in ([5, 1, 2, 33, 3], [1, 1, 1], [40, 1, 2, 16, 1, 1, 37]):
        t = sum(lens)
        x = _rand(t, channels + 40, seed=1, dtype=dtype)[:, 24: 24 + channels]
        w, bias = _rand(channels, taps, seed=2, scale=0.5, dtype=dtype), _rand(channels, seed=3, dtype=dtype)
        rows = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(5))[: len(lens)].tolist()
        start = _rand(len(lens) + 3, 11 + (taps - 1) * channels, seed=6)
        for b in (bias, None):
            res = []
            for impl in (ops, refs):
                state, out = start.clone(), torch.full((t, channels), float("nan"), device="cuda")
                impl.causal_conv_silu(x, w, state[:, 11:], FakeStep(lens, rows, device="cuda"), out, bias=b)
                res.append((out, state))
            torch.testing.assert_close(res[0][0], res[1][0], atol=2e-5, rtol=2e-5)
            assert torch.equal(res[0][1], res[1][1]), "the inputs are kept as they are, and foreign slots too"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, parts, width", [(1, 1, 8), (33, 4, 80), (7, 3, 515), (20, 2, 1024), (5, 1, 2048)])
def test_norm_behind_the_gate_kernel(dtype, rows, parts, width) -> None:
    ops = _ops()
    y, z = _rand(rows, parts, width, seed=1, scale=3.0), _rand(rows, parts * width + 9, seed=2, scale=2.0, dtype=dtype)[:, : parts * width]
    w = (1 + _rand(parts * width, seed=3, scale=0.3)).to(dtype)
    res = []
    for impl in (ops, refs):
        out = torch.empty(rows, parts * width, dtype=dtype, device="cuda")
        impl.head_norm_gate(y, w, True, z, True, 1e-6, out, gate_silu=True, gate_first=True)
        res.append(out.float())
    torch.testing.assert_close(res[0], res[1], atol=3e-2 if dtype == torch.bfloat16 else 3e-5, rtol=2e-2 if dtype == torch.bfloat16 else 3e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [8, 37, 1024])
def test_sinusoidal_embedding_kernel(dtype, hidden) -> None:
    """Positions from the first to far beyond any prompt; an id outside the table gives a row of NaN."""
    ops = _ops()
    table = _rand(30, hidden, seed=1, dtype=dtype)
    pos = torch.tensor([0, 1, 2, 255, 256, 4095, 65537, 1000003], dtype=torch.int32, device="cuda")
    ids = torch.tensor([3, 0, 29, 3, 7, 1, 1, 2], dtype=torch.int32, device="cuda")
    freq = (1e4 ** (-2.0 * torch.arange((hidden + 1) // 2, dtype=torch.float64) / hidden)).cuda()
    got, want = torch.empty(8, hidden, device="cuda"), torch.empty(8, hidden, device="cuda")
    ops.embed_pos_norm(ids, pos, table, None, None, 0.0, got, 1.7, freq=freq)
    refs.embed_pos_norm(ids, pos, table, None, None, 0.0, want, 1.7, freq=freq)
    torch.testing.assert_close(got, want, atol=3e-6, rtol=1e-6)
    bad = torch.empty(8, hidden, device="cuda")
    ops.embed_pos_norm(ids + 1, pos, table, None, None, 0.0, bad, 1.7, freq=freq)
    assert bool(bad[2].isnan().all()) and int(bad.isnan().any(1).sum()) == 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, hidden", [(1, 48), (37, 256), (5, 37), (300, 1024)])
def test_stream_beside_the_embedding_kernel(dtype, rows, hidden) -> None:
    ops = _ops()
    resid, first, delta = _rand(rows, hidden, seed=1, scale=5.0), _rand(rows, hidden, seed=2), _rand(rows, hidden, seed=3, dtype=dtype)
    for d in (delta, None):
        got, want = (torch.empty(rows, 2 * hidden, dtype=dtype, device="cuda") for _ in (0, 1))
        kept = resid.clone()
        ops.stream_beside(resid, d, first, got)
        refs.stream_beside(resid, d, first, want)
        assert torch.equal(got, want) and torch.equal(resid, kept)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, hidden, inner", [(1, 64, 80), (5, 72, 40), (8, 1024, 4096), (16, 256, 2048), (16, 3072, 1024), (64, 128, 256), (300, 320, 4096),
                                                 (2048, 1024, 4096), (777, 512, 2056), (130, 96, 200)])
def test_product_with_the_exact_gelu(dtype, rows, hidden, inner) -> None:
    """Few rows, tiles of the tcgen05 product (single and by pairs of CTAs) with ragged edges, and the library's product."""
    ops = _ops()
    if dtype == torch.float32 and rows > 1000:
        pytest.skip("the 32-bit product is the same kernel at every size")
    x, w = _rand(rows, hidden, seed=1, dtype=dtype), _rand(inner, hidden, seed=2, scale=1.5 * hidden ** -0.5, dtype=dtype)
    got, want = torch.full((rows, inner), float("nan"), dtype=dtype, device="cuda"), torch.empty(rows, inner, dtype=dtype, device="cuda")
    ops.gemm_activated(x, w, got, "gelu")
    refs.gemm_activated(x, w, want, "gelu")
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=1.6e-2)
    torch.testing.assert_close(got.float(), want.float(), **tol)


def test_gelu_of_the_epilogue_is_exact_to_its_rounding() -> None:
    """A product with a scaled unit matrix: every value of the range goes through the activation of the tcgen05 product."""
    ops = _ops()
    k = 256
    x = (torch.arange(4096 * k, dtype=torch.float64) / (4096 * k) * 16 - 8).view(4096, k).bfloat16().cuda()
    w = torch.zeros(2048, k, dtype=torch.bfloat16, device="cuda")
    w[:k] = torch.eye(k, dtype=torch.bfloat16, device="cuda")
    out = torch.empty(4096, 2048, dtype=torch.bfloat16, device="cuda")
    assert ops.tcgen05_tiles(4096, 2048, 256)
    ops.gemm_activated(x, w, out, "gelu")
    z = x.double()
    want = 0.5 * z * torch.special.erfc(-z / 2 ** 0.5)
    torch.testing.assert_close(out[:, :k].double(), want, rtol=2 ** -8, atol=1e-9)
    assert int(out[:, k:].count_nonzero()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("activation", ["silu", "gelu_tanh", "gelu"])
def test_activation_kernel(dtype, activation) -> None:
    ops = _ops()
    x = _rand(77, 130, seed=1, scale=3.0, dtype=dtype)
    got, want = x.clone(), x.clone()
    ops.activate(got, activation)
    refs.activate(want, activation)
    torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))


# ------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {k: write_model(tmp_path_factory.mktemp("risonex" + k), k) for k in CONFIGS}


LENGTHS = {"A": [1, 2, 9, 37, 70, 131], "B": [3, 33, 64, 97], "C": [5, 18, 40, 100], "D": [2, 47, 160]}


@pytest.fixture(scope="module")
def oracle(folders):
    out = {}
    for which in CONFIGS:
        vocab = plain.read_config(folders[which])["vocab"]
        reqs = {f"r{i}": random_prompt(n, vocab, 200 + 7 * i) for i, n in enumerate(LENGTHS[which])}
        out[which] = (reqs, {rid: plain_oracle(folders[which], toks) for rid, toks in reqs.items()})
    return out


def _check(got, reqs, want, dtype, what) -> list:
    assert all(sorted(got[rid]) == list(range(len(reqs[rid]))) for rid in got)
    rows = torch.cat([torch.stack([got[rid][p] for p in range(len(reqs[rid]))]) for rid in got])
    wanted, cond = torch.cat([want[rid][0] for rid in got]), torch.cat([want[rid][1] for rid in got])
    if dtype == torch.float32 or len(rows) >= 20:
        assert_rows_close(rows, wanted, cond, dtype, what)
    return [(rows, wanted, cond)]


def _close(parts, dtype, what) -> None:
    """All rows of several schedules together (a schedule of a handful of rows says little in bfloat16: one of them may
    have taken another expert)."""
    assert_rows_close(*(torch.cat(x) for x in zip(*parts)), dtype, what)


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
    every = []
    for n, steps in enumerate(plans):
        got, _ = run_steps(model, page, steps, cases.max_live_tokens(steps))
        every += _check(got, reqs, want, dtype, f"{which}, schedule {n}")
    _close(every, dtype, which)


@pytest.mark.parametrize("seed", list(range(1, 13)))
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
    """A prompt of several hundred tokens at the sizes of the tensor-core kernels: the scan of a long portion runs in
    segments, chunks pass over prompt and decoded tokens, a decoded token's keys are cut into ranges."""
    from tinyserve_b200.model import DecoderModel

    folder = write_model(tmp_path, CONFIG_D, 31)
    vocab = CONFIG_D["vocab"]
    reqs = {"long": random_prompt(420, vocab, 41), "short": random_prompt(9, vocab, 43)}
    assert _ops().linear_scan_segments(420, 1, 4, 64, 64)[1] > 1
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
    """2,048 tokens at width 1,024 through both layer kinds, both feed-forwards and a loop, experts in tiles of 128 sorted
    rows: two different prompts one after the other on the same scratch, overlap on and off, equal bit for bit."""
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.engine.replay import Replayer
    from tinyserve_b200.model import DecoderModel
    from risonex_cases import attention, config, dense, mamba, moe

    cfg = config(1000, 1024, 1.0, 1e-6, [(mamba(16, 2, 128, 64, 4, 2), dense(4096)), (attention(8, 4, 64, 128, 0.125, 0.2, 300), moe(14, 2, 3, 512, 512, 2.0))],
                 (0, 2, 2))
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
