"""Small Sanevik configurations that differ from one another in every size and option, a generator of random ones,
and helpers shared by the host-only and the GPU tests of that architecture."""

from __future__ import annotations

import random
from pathlib import Path

import torch

from diderax_cases import assert_rows_close as _assert_rows_close
from gasavik_cases import row_errors


def rot(dims, base, scaling=None):
    out = {"dims": dims, "base": base}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, scale, rotary, window):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotary}
    if window is not None:
        out["mask"] = {"size": window}
    return out


def pair(left, softcap, conv, right_heads, right_dim, right_vdim, right_rot, decay, left_scale, right_scale):
    return {"left": {**left, "softcap": softcap, "conv": conv},
            "right": {"heads": right_heads, "dim": right_dim, "vdim": right_vdim, "rot": right_rot, "decay": list(decay)},
            "left_scale": left_scale, "right_scale": right_scale}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


# A loop in the middle of the order that holds both kinds of layer; grouped heads, value heads of their own size, a
# partial rotation with scaling, windows of one page and of no multiple of anything; a layer without experts.
CONFIG_A = {
    "architecture": "Sanevik", "vocab": 101, "width": 64, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        {"type": "attention", "mixer": attention(4, 2, 32, 24, 0.2, rot(16, 1e4, (4.0, 64, 8.0, 1.0)), 19), "mlp": moe(5, 2, 24, 1.5)},
        {"type": "parallel", "mixer": pair(attention(4, 2, 16, 16, 0.25, rot(8, 1e3), 16), 5.0, 3, 2, 16, 24, rot(16, 1e4), (0.9, 0.99), 0.7, 1.3),
         "mlp": moe(4, 3, 16, 0.7)},
        {"type": "attention", "mixer": attention(2, 1, 16, 16, 0.3, rot(16, 5e4), 7), "mlp": None},
        {"type": "attention", "mixer": attention(3, 3, 16, 16, 0.25, rot(2, 100.0, (2.0, 4096, 32.0, 1.0)), 40), "mlp": moe(8, 1, 32, 3.0)},
    ],
}

# The whole order in the loop, one pass; a convolution of two taps and one of five; every expert picked; more heads than
# a multiple of anything; a window of one; key sizes that are no multiple of 16; a rotation of two elements.
CONFIG_B = {
    "architecture": "Sanevik", "vocab": 89, "width": 48, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 3, "times": 1},
    "layers": [
        {"type": "parallel", "mixer": pair(attention(5, 5, 8, 24, 0.4, rot(2, 1e4), 9), 2.0, 2, 3, 24, 8, rot(6, 1e3), (0.5, 0.95, 1.0), 1.2, 0.6),
         "mlp": moe(3, 3, 40, 1.0)},
        {"type": "attention", "mixer": attention(6, 2, 12, 20, 0.3, rot(12, 1e3, (8.0, 32, 4.0, 0.5)), 1), "mlp": moe(6, 2, 8, 2.0)},
        {"type": "parallel", "mixer": pair(attention(3, 1, 24, 8, 0.2, rot(24, 1e5), 33), 50.0, 5, 1, 40, 16, rot(40, 1e6), (0.97,), 0.5, 1.0),
         "mlp": None},
    ],
}

# One head everywhere, no loop, a convolution of one tap (no state of its own), one expert, attention without a window.
CONFIG_C = {
    "architecture": "Sanevik", "vocab": 61, "width": 32, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "parallel", "mixer": pair(attention(1, 1, 48, 40, 0.15, rot(32, 1e4), None), 8.0, 1, 1, 8, 8, rot(2, 50.0), (0.75,), 1.0, 1.0),
         "mlp": moe(1, 1, 24, 1.5)},
        {"type": "attention", "mixer": attention(1, 1, 40, 40, 0.2, rot(40, 300.0), None), "mlp": moe(2, 1, 16, 0.5)},
    ],
}

# Sizes at which the bfloat16 kernels run on the tensor cores: attention heads of 64 and 128, mixed heads of 64 and of
# 128 (more than 16 of them in one layer), experts as wide as a tile; a loop of three passes over one layer.
CONFIG_D = {
    "architecture": "Sanevik", "vocab": 211, "width": 128, "norm": {"eps": 1e-6}, "loop": {"start": 1, "stop": 2, "times": 3},
    "layers": [
        {"type": "parallel", "mixer": pair(attention(18, 9, 16, 32, 0.12, rot(16, 1e4), 50), 6.0, 4, 2, 64, 64, rot(64, 1e4), (0.9, 0.995), 0.5, 0.8),
         "mlp": moe(8, 2, 64, 2.0)},
        {"type": "attention", "mixer": attention(4, 2, 64, 64, 0.06, rot(32, 5e5, (4.0, 512, 16.0, 1.0)), 70), "mlp": moe(4, 2, 128, 1.5)},
        {"type": "parallel", "mixer": pair(attention(4, 2, 128, 128, 0.05, rot(128, 1e5), 37), 20.0, 2, 1, 128, 32, rot(64, 1e4), (0.98,), 0.9, 0.6),
         "mlp": moe(6, 1, 64, 7.0)},
        {"type": "attention", "mixer": attention(2, 1, 128, 128, 0.04, rot(128, 1e4), 128), "mlp": None},
    ],
}

CONFIGS = {"A": (CONFIG_A, 31), "B": (CONFIG_B, 32), "C": (CONFIG_C, 33), "D": (CONFIG_D, 34)}


def random_config(seed: int) -> dict:
    """A configuration with every size, constant, the layer order and the loop drawn at random."""
    rng = random.Random(seed)
    width = rng.choice([24, 40, 64, 72])

    def rotary(dim):
        scaling = None
        if rng.random() < 0.5:
            scaling = (rng.choice([1.0, 2.0, 8.0]), rng.choice([16, 128, 2048]), rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0]))
        return rot(rng.choice([2, dim // 2 // 2 * 2 or 2, dim]), rng.choice([100.0, 1e4, 5e5]), scaling)

    def attn():
        groups, dim = rng.randint(1, 3), rng.choice([8, 16, 24, 32, 64])
        return attention(groups * rng.randint(1, 3), groups, dim, rng.choice([dim, dim, 8, 16, 24]), rng.uniform(0.1, 0.4), rotary(dim),
                         rng.choice([1, 5, 8, 16, 21, 40, None]))

    layers = []
    for _ in range(rng.randint(2, 4)):
        kind = rng.choice(["attention", "parallel"])
        if kind == "attention":
            mixer = attn()
        else:
            left = attn()
            left["rot"].pop("scaling", None)
            heads, dim = rng.randint(1, 3), rng.choice([8, 16, 24, 40])
            right_rot = rotary(dim)
            right_rot.pop("scaling", None)
            mixer = pair(left, rng.choice([1.0, 5.0, 30.0]), rng.randint(1, 6), heads, dim, rng.choice([8, 16, 24]), right_rot,
                         [rng.choice([0.5, 0.9, 0.99, 1.0]) for _ in range(heads)], rng.uniform(0.3, 1.3), rng.uniform(0.3, 1.3))
        experts = rng.randint(1, 8)
        mlp = None if rng.random() < 0.25 else moe(experts, rng.randint(1, experts), rng.choice([8, 16, 40]), rng.choice([0.5, 2.0, 7.0]))
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    out = {"architecture": "Sanevik", "vocab": rng.randint(40, 150), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}
    if rng.random() < 0.75:
        start = rng.randint(0, len(layers) - 1)
        out["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return out


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
    import plain_sanevik as plain

    cfg = plain.read_config(folder)
    want = plain.forward(cfg, plain.read_weights(folder, torch.float64), tokens)
    low = plain.forward(cfg, plain.read_weights(folder, torch.float32), tokens).double()
    return want.float(), row_errors(low, want)


def assert_rows_close(rows: torch.Tensor, want: torch.Tensor, cond: torch.Tensor, dtype: torch.dtype, what: str = "") -> None:
    """float32: as for Diderax (a limit per position that grows with its conditioning: the retention's normed read-out
    loses the digits that cancel at a request's first tokens). bfloat16: a token whose best router logits lie closer
    together than the rounding of its input takes another expert than the oracle, and its row (and, diluted, rows that
    attend to it) differs by much more than rounding; so the rows are judged by their median and their upper quartile
    (a handful of rows by the median alone), and the float32 run of the same schedule carries the exactness."""
    if dtype == torch.float32:
        _assert_rows_close(rows, want, cond, dtype, what)
        return
    assert not rows.isnan().any(), f"{what}: NaN in the logits"
    err = row_errors(rows, want).sort().values
    median, upper = float(err[len(err) // 2]), float(err[(3 * len(err)) // 4])
    assert median < (0.05 if len(err) >= 20 else 0.15), f"{what}: median relative error {median:.3g} over {len(err)} rows"
    assert len(err) < 20 or upper < 0.12, f"{what}: upper quartile {upper:.3g} over {len(err)} rows"
