"""Sanevik on the host: its configuration and tensor names; the kernels' references against the plain
implementation, one mechanism at a time, with inputs made so that a fault shows; and the whole engine (cache
manager, step function, scheduler, sampler) with the references in the kernels' place against the plain model,
under every cut of the work."""

from __future__ import annotations

import copy
import json
import math
from dataclasses import replace

import pytest
import torch

import kernel_refs as refs
import plain_sanevik as plain
import replay_cases as cases
from fegilix_cases import FakeStep, run_steps
from guzovik_cases import FakeCtx
from kernel_refs import use_references
from sanevik_cases import CONFIGS, CONFIG_A, CONFIG_C, assert_rows_close, oracle as plain_oracle, random_config, rot, write_model
from tiny_configs import random_prompt

from tinyserve_b200.config import PartSpec, UnsupportedConfigError, config_from_dict
from tinyserve_b200.kernels.ops import RouteRule
from tinyserve_b200.model import DecoderModel, build_parts
from tinyserve_b200.parts import KVNeed, SplitKVNeed, StateNeed
from tinyserve_b200.parts.rope import RotaryEncoding
from tinyserve_b200.weights.loader import checkpoint_names, merge_specs


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {k: write_model(tmp_path_factory.mktemp("sanevik" + k), k) for k in CONFIGS}


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64) * scale


# ------------------------------------------------------------------ configuration
def test_config_round_trip_and_names(folders) -> None:
    for which, (cfg, _) in CONFIGS.items():
        c = config_from_dict(cfg)
        assert config_from_dict(c.to_dict()) == c
        assert json.loads((folders[which] / "config.json").read_text())["architecture"] == "Sanevik"
    names = checkpoint_names(merge_specs(build_parts(config_from_dict(CONFIG_A).to_spec()).tensor_specs()))
    assert names["embed"] == (101, 64) and names["final.norm"] == (64,) and names["loop.step"] == (2, 64) and "head" not in names
    assert names["l0.mix.q"] == (128, 64) and names["l0.mix.k"] == (64, 64) and names["l0.mix.v"] == (48, 64)
    assert names["l0.mix.sink"] == (4,) and names["l0.mix.o"] == (64, 96) and "l0.mix.q.conv" not in names
    assert names["l0.mlp.router"] == (5, 64) and names["l0.mlp.e4.down"] == (64, 24) and names["l0.norm2"] == (64,)
    left, right = "l1.mix.left.", "l1.mix.right."
    assert names[left + "q.conv"] == (64, 3) and names[left + "v.conv"] == (32, 3) and names[left + "talk"] == (4, 4)
    assert left + "sink" not in names and names[left + "o"] == (64, 64)
    assert names[right + "k"] == (32, 64) and names[right + "g"] == (48, 64) and names[right + "o"] == (64, 48)
    assert not any(n.startswith("l2.mlp.") or n == "l2.norm2" for n in names)
    assert "loop.step" not in checkpoint_names(merge_specs(build_parts(config_from_dict(CONFIG_C).to_spec()).tensor_specs()))


def test_order_and_cache_needs(folders) -> None:
    model = DecoderModel.from_folder(folders["A"], torch.float32, "cpu")
    assert [c.layer for c in model.spec.order] == [0, 1, 2, 1, 2, 3]
    inputs = [c.stream_input and (c.stream_input.args["index"], c.stream_input.args["add_origin"]) for c in model.spec.order]
    assert inputs == [None, (0, False), None, (1, True), None, None]
    pair = [KVNeed(2, 16, 16), StateNeed((2 * 128,), torch.float32), StateNeed((2 * 16 * 24,), torch.float32)]
    tail = KVNeed(1, 16, 7)
    assert model.cache_needs() == [SplitKVNeed(2, 32, 24, 19), *pair, tail, *pair, tail, KVNeed(3, 16, 40)]
    one_tap = DecoderModel.from_folder(folders["C"], torch.float32, "cpu").cache_needs()
    assert one_tap == [SplitKVNeed(1, 48, 40), StateNeed((64,), torch.float32), KVNeed(1, 40)]


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "has no 'slow'"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "positive values"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "must be positive"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("softcap"), "has no 'softcap'"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(conv=0), "conv at least 1"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]), "1 decay constants for 2 heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "only 'moe'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top=6 of 5 experts"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0), "must be positive"),
    (lambda c: c["loop"].update(stop=5), "does not fit 4 layers"),
    (lambda c: c["loop"].update(times=0), "does not fit"),
    (lambda c: c.pop("vocab"), "has no 'vocab'"),
])
def test_config_refusals(change, message) -> None:
    cfg = copy.deepcopy(CONFIG_A)
    change(cfg)
    with pytest.raises(UnsupportedConfigError, match=message):
        config_from_dict(cfg)


# ------------------------------------------- the references, one mechanism at a time
@pytest.mark.parametrize("dims, base, scaling", [(16, 1e4, (4.0, 64, 8.0, 1.0)), (48, 3e4, (2.0, 4096, 32.0, 1.0)), (2, 100.0, (8.0, 16, 4.0, 0.5)),
                                                 (64, 5e5, (1.0, 2048, 32.0, 1.0)), (8, 1e3, (3.0, 4, 32.0, 16.0))])
def test_yarn_frequencies_and_tables(dims, base, scaling) -> None:
    rotary = rot(dims, base, scaling)
    freq, mult = plain.frequencies(rotary)
    enc = RotaryEncoding(dims, dims, base, "interleaved", rotary["scaling"])
    torch.testing.assert_close(enc._inv_freq_host, torch.tensor(freq, dtype=torch.float64), rtol=1e-12, atol=0.0)
    assert enc.mult == pytest.approx(mult) and enc.key() != RotaryEncoding(dims, dims, base, "interleaved").key()
    pos = torch.tensor([0, 1, 77, 5000], dtype=torch.int32)
    cos, sin = torch.empty(4, dims // 2), torch.empty(4, dims // 2)
    refs.rope_tables(pos, enc._inv_freq_host, cos, sin, enc.mult)
    for i, p in enumerate(pos.tolist()):
        for j, f in enumerate(freq):
            assert float(cos[i, j]) == pytest.approx(mult * math.cos(p * f), abs=1e-6)
            assert float(sin[i, j]) == pytest.approx(mult * math.sin(p * f), abs=1e-6)


def test_the_ramp_lies_between_a_fast_and_a_slow_pair() -> None:
    """The fastest pairs keep their frequency, the slowest have it divided by the factor, one in between is neither."""
    rotary = rot(64, 1e4, (4.0, 4096, 32.0, 1.0))
    freq, _ = plain.frequencies(rotary)
    bare, _ = plain.frequencies(rot(64, 1e4))
    ratio = [a / b for a, b in zip(freq, bare)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(0.25) and any(0.3 < x < 0.9 for x in ratio)
    assert all(x >= y - 1e-12 for x, y in zip(ratio, ratio[1:]))


@pytest.mark.parametrize("taps, cuts", [(1, [9]), (2, [9]), (2, [1, 1, 7]), (3, [2, 2, 5]), (4, [4, 5]), (5, [1, 2, 6]), (7, [2, 1, 6])])
def test_reference_convolution_rotation_and_unit_norm(taps, cuts) -> None:
    heads, groups, d, dv, page, t = 4, 2, 8, 6, 4, 9
    channels = (heads + groups) * d + groups * dv
    u, w = _rand(t, channels + 3, seed=1), _rand(channels, taps, seed=2)
    rotary = rot(6, 100.0, (2.0, 32, 4.0, 1.0))
    enc = RotaryEncoding(d, 6, 100.0, "interleaved", rotary["scaling"])
    state = torch.zeros(3, (taps - 1) * channels, dtype=torch.float64)
    k_cache, v_cache = torch.zeros(3, groups, page, d, dtype=torch.float64), torch.zeros(3, groups, page, dv, dtype=torch.float64)
    slots = torch.tensor([8, 9, 10, 11, 0, 1, 2, 3, 4], dtype=torch.int32)
    q_out = torch.zeros(t, heads, d, dtype=torch.float64)
    at = 0
    for n in cuts:
        pos = torch.arange(at, at + n, dtype=torch.float64)
        ang = pos[:, None] * enc._inv_freq_host[None]
        part = torch.zeros(n, heads, d, dtype=torch.float64)
        refs.qkv_rotate(u[at: at + n], w.t().contiguous(), state, FakeStep([n], [1]), ang.cos() * enc.mult, ang.sin() * enc.mult, 6, True, 1e-5,
                        slots[at: at + n], k_cache, v_cache, page, heads, groups, d, dv, part)
        q_out[at: at + n] = part
        at += n
    y = plain.short_conv(u[:, :channels], w)
    want_q = plain.rms_norm(plain.rotate(y[:, : heads * d].reshape(t, heads, d), rotary, "interleaved"), None, 1e-5)
    want_k = plain.rms_norm(plain.rotate(y[:, heads * d: (heads + groups) * d].reshape(t, groups, d), rotary, "interleaved"), None, 1e-5)
    tol = dict(atol=2e-6, rtol=2e-6)                   # the reference convolves in 32-bit
    torch.testing.assert_close(q_out, want_q, **tol)
    for n in range(t):
        s = int(slots[n])
        torch.testing.assert_close(k_cache[s // page, :, s % page], want_k[n], **tol)
        torch.testing.assert_close(v_cache[s // page, :, s % page], y[n, (heads + groups) * d:].view(groups, dv), **tol)
    if taps > 1:
        torch.testing.assert_close(state[1], u[-(taps - 1):, :channels].reshape(-1)), "the last inputs of the convolution"
        assert state[0].abs().sum() == 0 and state[2].abs().sum() == 0


@pytest.mark.parametrize("heads, groups, window, cap, sink, mixed", [(4, 2, 5, 3.0, False, True), (3, 3, None, None, True, True), (6, 1, 1, 2.0, False, True),
                                                                     (2, 1, 12, 50.0, True, False)])
def test_reference_attention_with_mixed_heads(heads, groups, window, cap, sink, mixed) -> None:
    t, d, dv, page = 11, 6, 5, 4
    q, k, v = _rand(t, heads, d, seed=1, scale=2.0), _rand(t, groups, d, seed=2), _rand(t, groups, dv, seed=3)
    talk = _rand(heads, heads, seed=4) if mixed else None
    sinks = _rand(heads, seed=5) if sink else None
    want = plain.attention(q, k, v, 0.5, window, cap, None if sinks is None else sinks.tolist(), talk)
    table = torch.tensor([[2, 0, 1]], dtype=torch.int32)
    kc, vc = torch.zeros(3, groups, page, d, dtype=torch.float64), torch.zeros(3, groups, page, dv, dtype=torch.float64)
    for p in range(t):
        kc[table[0, p // page], :, p % page], vc[table[0, p // page], :, p % page] = k[p], v[p]
    for n in (t, 3, 1):
        out = torch.zeros(n, heads * dv, dtype=torch.float64)
        refs.talking_attention(q[t - n:], kc, vc, page, table, FakeCtx([n], [t]), 0.5, window or 0, cap, talk, out, sinks=sinks)
        torch.testing.assert_close(out.view(n, heads, dv), want[t - n:], atol=2e-6, rtol=2e-6)
    if mixed and heads > 1:
        plain_out = plain.attention(q, k, v, 0.5, window, cap, None if sinks is None else sinks.tolist(), None)
        assert (plain_out - want).abs().max() > 0.1


@pytest.mark.parametrize("cuts", [[13], [4, 9], [1, 1, 2, 9], [2] * 6 + [1]])
def test_reference_retention(cuts) -> None:
    heads, d, dv, width, t = 3, 8, 5, 20, 13
    m = {"heads": heads, "dim": d, "vdim": dv, "rot": rot(6, 50.0), "decay": [0.5, 0.97, 1.0]}
    h = _rand(t, width, seed=9)
    w = {"m." + n: _rand(*s, seed=i + 1, scale=0.5) for i, (n, s) in enumerate({
        "q": (24, width), "k": (24, width), "v": (15, width), "g": (15, width), "o": (width, 15)}.items())}
    q, k, v = h @ w["m.q"].T, h @ w["m.k"].T, h @ w["m.v"].T
    freq = torch.tensor(plain.frequencies(m["rot"])[0], dtype=torch.float64)
    state = torch.zeros(3, heads * d * dv, dtype=torch.float64)
    read = torch.zeros(t, heads, dv, dtype=torch.float64)
    at = 0
    for n in cuts:
        ang = torch.arange(at, at + n, dtype=torch.float64)[:, None] * freq[None]
        part = torch.zeros(n, heads, dv, dtype=torch.float64)
        refs.linear_scan_rotated(q[at: at + n], k[at: at + n], v[at: at + n], torch.tensor(m["decay"], dtype=torch.float64), ang.cos(), ang.sin(), 6, False,
                                 d ** -0.5, state, FakeStep([n], [1]), heads, d, dv, part)
        read[at: at + n] = part
        at += n
    gated = torch.zeros(t, heads * dv, dtype=torch.float64)
    refs.head_norm_gate(read, None, False, h @ w["m.g"].T, True, 1e-5, gated, gate_silu=True)
    torch.testing.assert_close(gated @ w["m.o"].T, plain.retention_mixer(h, w, "m.", m, 1e-5), atol=1e-5, rtol=1e-5)
    assert state[0].abs().sum() == 0 and state[2].abs().sum() == 0


@pytest.mark.parametrize("experts, top", [(8, 3), (5, 1), (4, 4), (1, 1)])
def test_reference_experts_with_weights_on_their_input(experts, top) -> None:
    t, width, ff, limit = 23, 12, 9, 0.8
    h = _rand(t, width, seed=1).float()
    w = {"m.router": _rand(experts, width, seed=2).float()}
    for e in range(experts):
        for i, (n, s) in enumerate({"gate": (ff, width), "up": (ff, width), "down": (width, ff)}.items()):
            w[f"m.e{e}.{n}"] = _rand(*s, seed=10 * e + i + 3).float()
    rule = RouteRule(scored=True, sigmoid=True, normalise=False, on_input=True)
    plan = refs.moe_route(h @ w["m.router"].T, top, None, rule=rule)
    want = plain.route(h, w, "m.", top)
    for n in range(t):
        assert plan["ids"].view(t, top)[n].tolist() == [e for e, _ in want[n]]
        assert plan["weights"].view(t, top)[n].tolist() == pytest.approx([x for _, x in want[n]], rel=1e-5)
    gu = torch.stack([torch.cat([w[f"m.e{e}.gate"], w[f"m.e{e}.up"]]) for e in range(experts)])
    down = torch.stack([w[f"m.e{e}.down"] for e in range(experts)])
    act, y, out = torch.zeros(t * top, ff), torch.zeros(t * top, width), torch.zeros(t, width)
    refs.moe_gemm(h, gu, act, plan, True, True, limit=limit)
    refs.moe_gemm(act, down, y, plan, False, False)
    refs.moe_combine(y, plan, None, out)
    mlp = {"router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    torch.testing.assert_close(out, plain.moe_ff(h, w, "m.", mlp), atol=1e-5, rtol=1e-5)
    outside = sum(x * plain.expert(h[:1], w, f"m.e{e}.", limit)[0] for e, x in want[0])
    assert (out[0] - outside).abs().max() > 1e-3, "a weight on the expert's output would give the same"


def test_reference_norm_that_folds_two_outputs_and_a_pass_vector() -> None:
    t, h = 5, 12
    resid, a, b, first = (_rand(t, h, seed=s).float() for s in (1, 2, 3, 4))
    vec, w = _rand(h, seed=5).float(), _rand(h, seed=6).float()
    x, out = resid.clone(), torch.zeros(t, h)
    refs.post_norm_add_rms_norm(x, a, None, None, 0.0, False, w, True, 1e-5, out, post_mult=0.7, second=b, second_scale=1.3,
                                add_rows=first, add_vec=vec)
    want = resid + 0.7 * a + 1.3 * b + first + vec
    torch.testing.assert_close(x, want)
    torch.testing.assert_close(out, plain.rms_norm(want, w, 1e-5), atol=1e-5, rtol=1e-5)


def test_a_stream_input_in_front_of_a_norm_that_does_not_add_it_is_refused() -> None:
    spec = config_from_dict(CONFIG_A).to_spec()
    layer = spec.layers[1]
    norm = PartSpec("rms_norm", {**layer.parts["mixer_norm"].args, "unit_offset": False})
    bad = replace(layer, parts={**layer.parts, "mixer_norm": norm})
    with pytest.raises(ValueError, match="does not add it"):
        build_parts(replace(spec, layers=(spec.layers[0], bad, *spec.layers[2:])))


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


def test_each_pass_has_caches_of_its_own_and_the_step_vectors_matter(folders) -> None:
    """Swapping the pass vectors, or leaving the embedding output out, changes the logits."""
    model = DecoderModel.from_folder(folders["A"], torch.float32, "cpu")
    toks = random_prompt(20, 101, 3)

    def last():
        with use_references():
            got, _ = run_steps(model, 4, cases.tail_decoded("a", toks, 8), 64)
        return got["a"][len(toks) - 1]

    base = last()
    model.tensors["loop.step"].copy_(model.tensors["loop.step"].flip(0).clone())
    assert (last() - base).abs().max() > 1e-3
    model.tensors["loop.step"].copy_(model.tensors["loop.step"].flip(0).clone())
    torch.testing.assert_close(last(), base)
    model.parts.stream_inputs[3].needs_origin = False
    assert (last() - base).abs().max() > 1e-3


def test_greedy_generation_through_the_engine_on_host(folders) -> None:
    from tinyserve_b200.cache import CacheManager
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
