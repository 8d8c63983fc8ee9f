"""Risonex on the host: its configuration and tensor names; the page table of chunked attention; the kernels'
references against the plain implementation, one mechanism at a time, with inputs made so that a fault shows; and the
whole engine (cache manager, step function, scheduler, sampler) with the references in the kernels' place against the
plain model, under every cut of the work."""

from __future__ import annotations

import copy
import json
import math

import pytest
import torch

import kernel_refs as refs
import plain_risonex as plain
import replay_cases as cases
from fegilix_cases import FakeStep, run_steps
from guzovik_cases import FakeCtx
from kernel_refs import use_references
from risonex_cases import CONFIGS, CONFIG_A, CONFIG_B, CONFIG_C, assert_rows_close, oracle as plain_oracle, random_config, write_model
from tiny_configs import random_prompt

from tinyserve_b200.cache import CacheManager
from tinyserve_b200.cache.allocator import PageAllocator
from tinyserve_b200.cache.block_table import BlockTable
from tinyserve_b200.config import UnsupportedConfigError, config_from_dict
from tinyserve_b200.kernels.ops import RouteRule
from tinyserve_b200.model import DecoderModel, build_parts
from tinyserve_b200.parts import KVNeed, SplitKVNeed, StateNeed
from tinyserve_b200.parts.attention import DifferentialAttention
from tinyserve_b200.parts.recurrent import StateSpaceMixer
from tinyserve_b200.weights.loader import checkpoint_names, merge_specs


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {k: write_model(tmp_path_factory.mktemp("risonex" + k), k) for k in CONFIGS}


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64) * scale


# ------------------------------------------------------------------ configuration
def test_config_round_trip_and_names(folders) -> None:
    for which, (cfg, _) in CONFIGS.items():
        c = config_from_dict(cfg)
        assert config_from_dict(c.to_dict()) == c
        assert json.loads((folders[which] / "config.json").read_text())["architecture"] == "Risonex"
    names = checkpoint_names(merge_specs(build_parts(config_from_dict(CONFIG_A).to_spec()).tensor_specs()))
    assert names["embed"] == (101, 64) and names["head"] == (101, 64) and names["final.norm"] == (64,) and names["loop.in"] == (64, 128)
    assert names["l0.mix.q"] == (128, 64) and names["l0.mix.k"] == (64, 64) and names["l0.mix.v"] == (64, 64) and names["l0.mix.o"] == (64, 128)
    assert names["l0.mix.q.norm"] == (16,) and names["l0.mix.lq1"] == names["l0.mix.lk2"] == (16,)
    assert names["l0.mlp.up"] == (88, 64) and names["l0.mlp.down"] == (64, 88) and "l0.mlp.gate" not in names
    assert names["l1.mix.in"] == (2 * 96 + 2 * 32 + 4, 64) and names["l1.mix.conv"] == (160, 3) and names["l1.mix.conv.b"] == (160,)
    assert names["l1.mix.dt_bias"] == names["l1.mix.A_log"] == names["l1.mix.D"] == (4,) and names["l1.mix.norm"] == (96,)
    assert names["l1.mix.o"] == (64, 96) and names["l1.mlp.router"] == (7, 64) and names["l1.mlp.correction"] == (7,)
    assert names["l1.mlp.e4.down"] == (64, 24) and "l1.mlp.e5.down" not in names and names["l1.mlp.shared.sg"] == (1, 64)
    assert not any(n.startswith("l2.mlp.") or n == "l2.norm2" for n in names) and "l3.mlp.shared.sg" not in names
    assert "loop.in" not in checkpoint_names(merge_specs(build_parts(config_from_dict(CONFIG_C).to_spec()).tensor_specs()))


def test_order_and_cache_needs(folders) -> None:
    model = DecoderModel.from_folder(folders["A"], torch.float32, "cpu")
    assert [c.layer for c in model.spec.order] == [0, 1, 2, 1, 2, 3]
    assert [c.stream_input is not None for c in model.spec.order] == [False, True, False, True, False, False]
    first, pair = KVNeed(2, 32, chunk=19), [StateNeed((4 * 16 * 24 + 2 * 160,), torch.float32), KVNeed(1, 48, chunk=40)]
    assert model.cache_needs() == [first, *pair, *pair, StateNeed((6 * 24 * 8 + 3 * 192,), torch.float32)]
    needs = DecoderModel.from_folder(folders["B"], torch.float32, "cpu").cache_needs()
    assert needs[0] == StateNeed((3 * 40 * 12,), torch.float32), "one tap keeps nothing"
    assert needs[1:3] == [SplitKVNeed(3, 24, 20, chunk=1), SplitKVNeed(5, 16, 24, chunk=33)]


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "has no 'diff'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "must be positive"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "not a multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "does not divide 4 x 24"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "must be at least 1"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "has no 'state'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "'dense' and 'moe'"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=8), "top=8 of 5 experts and 2 identity"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "must be positive"),
    (lambda c: c["loop"].update(stop=5), "does not fit 4 layers"),
    (lambda c: c["loop"].update(times=0), "does not fit"),
    (lambda c: c.pop("vocab"), "has no 'vocab'"),
])
def test_config_refusals(change, message) -> None:
    cfg = copy.deepcopy(CONFIG_A)
    change(cfg)
    with pytest.raises(UnsupportedConfigError, match=message):
        config_from_dict(cfg)


def test_parts_refuse_sizes_they_cannot_run() -> None:
    with pytest.raises(ValueError, match="or neither"):
        DifferentialAttention("m.", 8, 2, 1, 4, 8, 1.0, 0.2, 1e-5, window=4, chunk=4)
    with pytest.raises(ValueError, match="up to 256"):
        DifferentialAttention("m.", 8, 2, 1, 257, 8, 1.0, 0.2, 1e-5)
    with pytest.raises(ValueError, match="key size 300"):
        StateSpaceMixer("m.", 8, 2, 1, 300, 8, 2, 1, 1e-5)


# --------------------------------------------------------------- pages of a chunk
@pytest.mark.parametrize("chunk, page", [(8, 4), (10, 4), (3, 4), (1, 4), (16, 16), (7, 8), (64, 8)])
def test_pages_of_finished_chunks_are_given_back(chunk, page) -> None:
    """After every step the pages that hold a position of the next query's chunk are there, and no page before them."""
    for cuts in ([1] * 40, [5, 1, 9, 2, 20, 3], [37]):
        alloc = PageAllocator(64)
        table = BlockTable(alloc, page, chunk=chunk)
        n = 0
        for c in cuts:
            first = n // chunk * chunk
            table.append(c)
            for p in range(first, n + c):
                assert table.slot(p) >= 0
            n += c
            table.release_passed()
            assert all((table.pages[i] == -1) == ((i + 1) * page <= n // chunk * chunk) for i in range(len(table.pages)))
        table.release()
        assert alloc.num_used == 0


def test_a_chunk_group_gets_only_the_pages_its_requests_can_hold() -> None:
    needs = [KVNeed(1, 8, chunk=20), KVNeed(1, 8)]
    cache = CacheManager(needs, page_size=4, num_pages=100, max_requests=2, dtype=torch.float32, device="cpu", max_step_tokens=12)
    assert [g.num_pages for g in cache.groups] == [2 * 9, 100]
    assert cache.groups[0].most_pages_of(1000, 12) == 9 and cache.groups[1].most_pages_of(1000, 12) == 250
    assert cache.capacity_tokens == 400


# ------------------------------------------- the references, one mechanism at a time
@pytest.mark.parametrize("heads, groups, d, dv, chunk", [(4, 2, 3, 6, 5), (3, 3, 4, 5, 1), (2, 1, 6, 12, None), (6, 2, 2, 7, 12)])
def test_reference_differential_attention(heads, groups, d, dv, chunk) -> None:
    """Weights made so that neither map dominates; the factor, the order of the maps and the chunk all show."""
    t, width, page, eps = 13, 18, 4, 1e-5
    m = {"heads": heads, "kv_heads": groups, "dim": d, "vdim": dv, "scale": 0.8, "diff": 0.4, **({"mask": {"size": chunk}} if chunk else {})}
    w = {"m." + n: _rand(*s, seed=i + 1, scale=0.6).float() for i, (n, s) in enumerate({
        "q": (heads * 2 * d, width), "k": (groups * 2 * d, width), "v": (groups * dv, width), "o": (width, heads * dv), "q.norm": (d,), "k.norm": (d,),
        "lq1": (d,), "lk1": (d,), "lq2": (d,), "lk2": (d,)}.items())}
    h = _rand(t, width, seed=77).float()
    want = plain.attention_mixer(h, w, "m.", m, eps)
    part = DifferentialAttention("m.", width, heads, groups, d, dv, 0.8, 0.4, eps, chunk=chunk)
    part.bind("", {**w, "m.qkv": torch.cat([w["m.q"], w["m.k"], w["m.v"]])})
    assert float(part.factor) == pytest.approx(float(plain.mix_factor(w, "m.", 0.4)), rel=1e-5)
    table = torch.tensor([[2, 0, 3, 1]], dtype=torch.int32)
    for cuts in ([13], [1] * 13, [2, 7, 4]):
        kc, vc = torch.full((4, groups, page, 2 * d), float("nan")), torch.full((4, groups, page, dv), float("nan"))
        rows, at = [], 0
        for n in cuts:
            pos = torch.arange(at, at + n)
            ctx = FakeCtx([n], [at + n])
            ctx.slots = table[0].long()[pos // page] * page + pos % page
            rows.append(_attend(part, h[at: at + n], ctx, kc, vc, page, table))
            at += n
        torch.testing.assert_close(torch.cat(rows), want, atol=2e-5, rtol=2e-5)
    plain_mask = plain.attention_mixer(h, w, "m.", {**m, "mask": {"size": (chunk or 99) + 1}}, eps)
    assert chunk is None or (plain_mask - want).abs().max() > 1e-2
    if chunk == 1:
        return                  # a single key: both maps give its value, and only the factor's sign is left
    swapped = {**w, "m.lq1": w["m.lq2"], "m.lk1": w["m.lk2"], "m.lq2": w["m.lq1"], "m.lk2": w["m.lk1"]}
    assert (plain.attention_mixer(h, swapped, "m.", m, eps) - want).abs().max() > 1e-2


def _attend(part, h, ctx, kc, vc, page, table):
    """The mixer's forward with the references, on caches made by hand."""
    from types import SimpleNamespace

    from tinyserve_b200.parts import KVCacheEntry, KVGroupContext

    ctx.kv = {0: KVGroupContext(page, table, ctx.slots.int())}
    ctx.arena = SimpleNamespace(take=lambda shape, dtype: torch.full(shape, float("nan"), dtype=dtype))
    ctx.dtype = h.dtype
    with use_references():
        return part.forward(h, ctx, KVCacheEntry(0, kc, vc, page), True, None)


@pytest.mark.parametrize("taps, cuts", [(1, [13]), (2, [1, 1, 11]), (3, [2, 2, 9]), (4, [1] * 13), (7, [3, 1, 9])])
@pytest.mark.parametrize("heads, groups, n, dv, parts", [(4, 2, 5, 6, 3), (3, 3, 4, 5, 1), (2, 1, 7, 4, 8)])
def test_reference_state_space_mixer(taps, cuts, heads, groups, n, dv, parts) -> None:
    """Step sizes and rates spread widely, so that a decay, a step or a skip that is wrong shows."""
    from types import SimpleNamespace

    from tinyserve_b200.parts import StateCacheEntry

    t, width, eps = 13, 20, 1e-5
    inner, ch = heads * dv, heads * dv + 2 * groups * n
    m = {"heads": heads, "groups": groups, "state": n, "vdim": dv, "conv": taps, "norm_groups": parts}
    shapes = {"in": (inner + ch + heads, width), "conv": (ch, taps), "conv.b": (ch,), "dt_bias": (heads,), "A_log": (heads,), "D": (heads,),
              "norm": (inner,), "o": (width, inner)}
    w = {"m." + k: _rand(*s, seed=i + 1, scale=0.5 if k != "A_log" else 1.5).float() for i, (k, s) in enumerate(shapes.items())}
    h = _rand(t, width, seed=9).float()
    want = plain.mamba2_mixer(h, w, "m.", m, eps)
    part = StateSpaceMixer("m.", width, heads, groups, n, dv, taps, parts, eps)
    part.bind("", w)
    state = torch.zeros(3, *part.cache_need().shape)
    rows, at = [], 0
    for c in cuts:
        ctx = FakeStep([c], [1])
        ctx.dtype, ctx.max_query_len = torch.float32, c
        ctx.arena = SimpleNamespace(take=lambda shape, dtype: torch.full(shape, float("nan"), dtype=dtype))
        with use_references():
            rows.append(part.forward(h[at: at + c], ctx, StateCacheEntry(state), True, None))
        at += c
    torch.testing.assert_close(torch.cat(rows), want, atol=3e-5, rtol=3e-5)
    assert state[0].abs().sum() == 0 and state[2].abs().sum() == 0
    if parts > 1:
        other = plain.mamba2_mixer(h, w, "m.", {**m, "norm_groups": 1}, eps)
        assert (other - want).abs().max() > 1e-2, "parts normed together would give the same"


def test_gated_before_it_is_normed() -> None:
    y, z, w = _rand(3, 12, seed=1).float(), _rand(3, 12, seed=2).float(), _rand(12, seed=3).float()
    out, late = torch.zeros(3, 12), torch.zeros(3, 12)
    refs.head_norm_gate(y.view(3, 3, 4), w, True, z, True, 1e-5, out, gate_silu=True, gate_first=True)
    torch.testing.assert_close(out, plain.gate_and_norm(y, z, w, 3, 1e-5), atol=1e-5, rtol=1e-5)
    refs.head_norm_gate(y.view(3, 3, 4), w, True, z, True, 1e-5, late, gate_silu=True)
    assert (late - out).abs().max() > 0.1


@pytest.mark.parametrize("width", [6, 7, 40])
def test_reference_sinusoids(width) -> None:
    table, toks = _rand(9, width, seed=1), [3, 0, 8, 8, 1]
    freq = 1e4 ** (-2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width)
    out = torch.zeros(5, width)
    refs.embed_pos_norm(torch.tensor(toks), torch.arange(5), table.float(), None, None, 0.0, out, 2.5, freq=freq)
    want = plain.embedding({"embedding": {"scale": 2.5}, "width": width}, {"embed": table}, toks)
    torch.testing.assert_close(out, want.float(), atol=1e-5, rtol=1e-5)
    far = torch.zeros(1, width)
    refs.embed_pos_norm(torch.tensor([0]), torch.tensor([70000]), table.float() * 0, None, None, 0.0, far, 1.0, freq=freq)
    assert float(far[0, 1]) == pytest.approx(math.cos(70000.0), abs=1e-6)


@pytest.mark.parametrize("experts, identity, top, shared", [(5, 2, 3, 6), (4, 0, 4, None), (1, 3, 2, 4), (6, 1, 1, 9)])
def test_reference_experts(experts, identity, top, shared) -> None:
    t, width, ff = 23, 12, 9
    h = _rand(t, width, seed=1).float()
    w = {"m.router": _rand(experts + identity, width, seed=2).float(), "m.correction": _rand(experts + identity, seed=3, scale=0.3).float()}
    for e in [f"e{i}" for i in range(experts)] + (["shared"] if shared else []):
        inner = shared if e == "shared" else ff
        for i, (n, s) in enumerate({"gate": (inner, width), "up": (inner, width), "down": (width, inner)}.items()):
            w[f"m.{e}.{n}"] = _rand(*s, seed=10 * (experts if e == "shared" else int(e[1:])) + i + 7, scale=0.5).float()
    mlp = {"router": {"experts": experts, "identity": identity, "top": top, "scale": 1.7}}
    gate = None
    if shared:
        w["m.shared.sg"], mlp["shared"] = _rand(1, width, seed=5).float(), {"ff": shared}
        gate = (h @ w["m.shared.sg"].T).reshape(-1)
    rule = RouteRule(scored=True, scale=1.7, identity=identity, correction=w["m.correction"])
    plan = refs.moe_route(h @ w["m.router"].T, top, None, rule=rule)
    gu = torch.stack([torch.cat([w[f"m.e{e}.gate"], w[f"m.e{e}.up"]]) for e in range(experts)])
    act, y, out = torch.zeros(t * top, ff), torch.zeros(t * top, width), torch.zeros(t, width)
    refs.moe_gemm(h, gu, act, plan, True, True)
    refs.moe_gemm(act, torch.stack([w[f"m.e{e}.down"] for e in range(experts)]), y, plan, False, False)
    refs.moe_combine(y, plan, plain.expert(h, w, "m.shared.") if shared else None, out, x=h if identity else None, shared_gate=gate)
    torch.testing.assert_close(out, plain.moe_ff(h, w, "m.", mlp), atol=1e-4, rtol=1e-4)


def test_reference_plain_feed_forward_has_the_exact_gelu() -> None:
    h, up, down = _rand(9, 6, seed=1).float(), _rand(10, 6, seed=2).float(), _rand(6, 10, seed=3).float()
    act = torch.zeros(9, 10)
    refs.gemm_activated(h, up, act, "gelu")
    torch.testing.assert_close(act @ down.T, plain.dense_ff(h, {"m.up": up, "m.down": down}, "m."), atol=1e-5, rtol=1e-5)
    tanh = torch.zeros(9, 10)
    refs.gemm_activated(h, up, tanh, "gelu_tanh")
    assert (tanh - act).abs().max() > 1e-4


# ----------------------------------------------- the engine on the host, every cut
LENGTHS = {"A": [1, 2, 9, 37, 70], "B": [3, 45, 80], "C": [5, 18, 40], "D": [2, 21, 60]}


@pytest.fixture(scope="module")
def oracle(folders):
    out = {}
    for which in CONFIGS:
        vocab = plain.read_config(folders[which])["vocab"]
        reqs = {f"r{i}": random_prompt(n, vocab, 100 + 7 * i) for i, n in enumerate(LENGTHS[which])}
        out[which] = (reqs, {rid: plain_oracle(folders[which], toks) for rid, toks in reqs.items()})
    return out


@pytest.mark.parametrize("which, page", [("A", 4), ("A", 16), ("B", 8), ("C", 4), ("D", 16)])
def test_engine_on_host_under_every_cut(folders, oracle, which, page) -> None:
    reqs, want = oracle[which]
    model = DecoderModel.from_folder(folders[which], torch.float32, "cpu")
    plans = [cases.mixed(reqs, 3), cases.mixed(reqs, 5, max_live=2)]
    for rid, toks in reqs.items():
        plans += [cases.whole(rid, toks), cases.tail_decoded(rid, toks, 12), cases.portions(rid, toks, 1)]
    with use_references():
        for steps in plans:
            got, _ = run_steps(model, page, steps, cases.max_live_tokens(steps))
            for rid in got:
                rows = torch.stack([got[rid][p] for p in range(len(reqs[rid]))])
                assert_rows_close(rows, *want[rid], torch.float32, f"{which}/{rid}")


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_configurations_drawn_at_random_on_host(seed, tmp_path) -> None:
    cfg = random_config(seed)
    folder = write_model(tmp_path, cfg, seed)
    reqs = {f"r{i}": random_prompt(n, cfg["vocab"], 10 * seed + i) for i, n in enumerate((1, 14, 47))}
    want = {rid: plain_oracle(folder, toks) for rid, toks in reqs.items()}
    model = DecoderModel.from_folder(folder, torch.float32, "cpu")
    with use_references():
        for steps in (cases.mixed(reqs, seed), cases.portions("r2", reqs["r2"], seed)):
            got, _ = run_steps(model, 8, steps, cases.max_live_tokens(steps))
            for rid in got:
                assert_rows_close(torch.stack([got[rid][p] for p in range(len(reqs[rid]))]), *want[rid], torch.float32, f"{seed}/{rid}")


def test_the_product_in_front_of_every_pass_reads_the_stream_and_the_embedding(folders) -> None:
    """Either half of the matrix set to zero changes the logits, and so does one pass less."""
    toks = random_prompt(20, 101, 3)

    def last(model):
        with use_references():
            got, _ = run_steps(model, 4, cases.tail_decoded("a", toks, 8), 64)
        return got["a"][len(toks) - 1]

    model = DecoderModel.from_folder(folders["A"], torch.float32, "cpu")
    base = last(model)
    kept = model.tensors["loop.in"].clone()
    for half in (slice(0, 64), slice(64, 128)):
        model.tensors["loop.in"][:, half] = 0
        assert (last(model) - base).abs().max() > 1e-3
        model.tensors["loop.in"].copy_(kept)
    torch.testing.assert_close(last(model), base)


def test_greedy_generation_through_the_engine_on_host(folders) -> None:
    from tinyserve_b200.engine import Engine

    cfg, w = plain.read_config(folders["B"]), plain.read_weights(folders["B"], torch.float64)
    prompts = [random_prompt(n, cfg["vocab"], 40 + n) for n in (3, 11, 26)]
    want = [plain.greedy(cfg, w, p, 6) for p in prompts]
    model = DecoderModel.from_folder(folders["B"], torch.float32, "cpu")
    for kw in (dict(num_pages=64), dict(num_pages=64, max_batch_tokens=8, chunked_prefill=True), dict(num_pages=6)):
        pages = kw.pop("num_pages")
        cache = CacheManager(model.cache_needs(), page_size=8, num_pages=pages, max_requests=3, dtype=torch.float32, device="cpu")
        with use_references():
            e = Engine(model, cache, max_num_seqs=3, **kw)
            assert e.generate(prompts, 6) == want
        assert all(g.allocator.num_used == 0 for g in cache.groups)
    assert len({tuple(x) for x in want}) > 1
