"""Small Risonex configurations that differ from one another in every size and option, a generator of random ones,
and helpers shared by the host-only and the GPU tests of that architecture."""

from __future__ import annotations

import random
from pathlib import Path

import torch

from diderax_cases import assert_rows_close as _assert_rows_close32
from gasavik_cases import row_errors


def attention(heads, kv_heads, dim, vdim, scale, diff, chunk):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if chunk is not None:
        out["mask"] = {"size": chunk}
    return out


def mamba(heads, groups, state, vdim, conv, norm_groups):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, shared, scale=None):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if scale is not None:
        router["scale"] = scale
    out = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def config(vocab, width, scale, eps, layers, loop=None):
    out = {"architecture": "Risonex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
           "layers": [{"type": "mamba2" if "state" in m else "attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# A loop in the middle of the order over both kinds of layer; grouped heads; values twice as wide as a map; chunks that
# are no multiple of a page; a layer without a feed-forward.
CONFIG_A = config(101, 64, 3.0, 1e-5, [
    (attention(4, 2, 16, 32, 0.3, 0.2, 19), dense(88)),
    (mamba(4, 2, 16, 24, 3, 4), moe(5, 2, 2, 24, 40, 1.5)),
    (attention(2, 1, 24, 48, 0.25, 0.5, 40), None),
    (mamba(6, 3, 24, 8, 4, 1), moe(4, 1, 3, 16, None)),
], (1, 3, 2))

# The whole order in the loop, one pass; value sizes unrelated to the maps'; a chunk of one; a convolution of one tap
# (nothing of it is state) and one of six; every router output picked; no identity experts.
CONFIG_B = config(89, 48, 1.0, 1e-6, [
    (mamba(3, 1, 40, 12, 1, 3), dense(40)),
    (attention(6, 3, 12, 20, 0.4, 0.0, 1), moe(3, 0, 3, 40, 24, 0.7)),
    (attention(5, 5, 8, 24, 0.35, 0.7, 33), moe(2, 2, 4, 8, 16, 2.0)),
    (mamba(8, 8, 8, 16, 6, 2), None),
], (0, 4, 1))

# One head everywhere, no loop, attention without chunks, one expert and one identity expert.
CONFIG_C = config(61, 32, 5.5, 1e-5, [
    (attention(1, 1, 20, 40, 0.2, 0.35, None), moe(1, 1, 1, 24, 8, 1.0)),
    (mamba(1, 1, 48, 40, 2, 1), dense(24)),
])

# Sizes at which the bfloat16 kernels run on the tensor cores: maps of 64 over values of 128 and of 32 over 64; experts
# as wide as a tile; a loop of three passes over the last two layers.
CONFIG_D = config(211, 128, 2.0, 1e-6, [
    (mamba(4, 2, 64, 64, 4, 2), dense(256)),
    (attention(4, 2, 64, 128, 0.12, 0.3, 70), moe(8, 2, 3, 64, 128, 2.0)),
    (attention(4, 4, 32, 64, 0.2, 0.6, 48), moe(4, 0, 2, 128, None, 1.5)),
    (attention(4, 1, 64, 128, 0.1, 0.1, None), dense(128)),
], (2, 4, 3))

CONFIGS = {"A": (CONFIG_A, 41), "B": (CONFIG_B, 42), "C": (CONFIG_C, 43), "D": (CONFIG_D, 44)}


def random_config(seed: int) -> dict:
    """A configuration with every size, constant, the layer order and the loop drawn at random."""
    rng = random.Random(seed)
    width = rng.choice([24, 40, 64, 72])
    layers = []
    for _ in range(rng.randint(2, 4)):
        if rng.random() < 0.5:
            groups, dim = rng.randint(1, 3), rng.choice([4, 8, 12, 16, 24, 32, 64])
            mixer = attention(groups * rng.randint(1, 3), groups, dim, rng.choice([2 * dim, 2 * dim, dim, 8, 20]), rng.uniform(0.1, 0.5),
                              rng.choice([0.0, 0.2, 0.45, 0.8]), rng.choice([1, 5, 8, 16, 21, 40, None]))
        else:
            groups = rng.randint(1, 3)
            heads, vdim = groups * rng.randint(1, 3), rng.choice([4, 8, 16, 20, 40])
            parts = rng.choice([n for n in range(1, heads * vdim + 1) if heads * vdim % n == 0 and heads * vdim // n >= 8 or n == 1])
            mixer = mamba(heads, groups, rng.choice([4, 8, 16, 20, 48]), vdim, rng.randint(1, 6), parts)
        kind = rng.random()
        if kind < 0.2:
            mlp = None
        elif kind < 0.5:
            mlp = dense(rng.choice([16, 40, 100]))
        else:
            experts, identity = rng.randint(1, 8), rng.randint(0, 3)
            mlp = moe(experts, identity, rng.randint(1, experts + identity), rng.choice([8, 16, 40]), rng.choice([None, 8, 24, 32]),
                      rng.choice([None, 0.5, 2.2]))
        layers.append((mixer, mlp))
    loop = None
    if rng.random() < 0.8:
        start = rng.randint(0, len(layers) - 1)
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return config(rng.randint(40, 150), width, rng.choice([1.0, 4.0, 10.0]), rng.choice([1e-5, 1e-6]), layers, loop)


def write_model(folder: Path, which: "str | dict", seed: int | None = None, std_scale: float = 6.0) -> Path:
    """The configuration with random weights, through the framework's random-weights mode."""
    import tinyserve_b200.architectures  # noqa: F401
    from tinyserve_b200.config import config_from_dict
    from tinyserve_b200.weights import write_random_model

    cfg, s = CONFIGS[which] if isinstance(which, str) else (which, seed)
    return write_random_model(folder, config_from_dict(cfg), s, torch.bfloat16, std_scale=std_scale)


def oracle(folder: Path, tokens: list[int]) -> tuple[torch.Tensor, torch.Tensor]:
    """The plain model's logits in 64-bit, and for every position how far the same plain model in 32-bit lies from
    them (its conditioning)."""
    import plain_risonex as plain

    cfg = plain.read_config(folder)
    want = plain.forward(cfg, plain.read_weights(folder, torch.float64), tokens)
    low = plain.forward(cfg, plain.read_weights(folder, torch.float32), tokens).double()
    return want.float(), row_errors(low, want)


def assert_rows_close(rows: torch.Tensor, want: torch.Tensor, cond: torch.Tensor, dtype: torch.dtype, what: str = "") -> None:
    """float32: a limit per position that grows with its conditioning. bfloat16: a token whose best router logits lie closer
    together than the rounding of its input takes another expert than the oracle, and its row (and, diluted, later rows)
    differs by much more than rounding; so the rows are judged by their median and their upper quartile (a handful of rows
    by the median alone), both with an allowance for the conditioning of such rows, carried from 32-bit to 16-bit rounding
    (a norm over a few columns, or over two maps that nearly cancel, magnifies it); the float32 run of the same schedule
    carries the exactness."""
    if dtype == torch.float32:
        _assert_rows_close32(rows, want, cond, dtype, what)
        return
    assert not rows.isnan().any(), f"{what}: NaN in the logits"
    err, amplified = row_errors(rows, want).sort().values, (cond * 2.0 ** 16).sort().values
    mid, up = len(err) // 2, (3 * len(err)) // 4
    few = len(err) < 20
    limit = (0.15 if few else 0.05) + 0.5 * float(amplified[mid])
    assert float(err[mid]) < limit, f"{what}: median relative error {float(err[mid]):.3g} over {len(err)} rows (limit {limit:.3g})"
    limit = 0.12 + 0.5 * float(amplified[up])
    assert few or float(err[up]) < limit, f"{what}: upper quartile {float(err[up]):.3g} over {len(err)} rows (limit {limit:.3g})"
