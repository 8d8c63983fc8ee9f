"""A plain, slow implementation of the Risonex decoder, one function per mechanism, written from the
design's equations and sharing no code with the product path. Everything runs token by token or
with full matrices on the CPU in one floating type (float64 for an oracle, float32 otherwise);
nothing is cached between calls.

Notation: ``h`` is a sub-layer's input ``[T, width]``; weights are ``[out, in]``; ``w`` maps tensor
names to tensors already converted to the working type; ``p`` is a tensor-name prefix; ``m`` is a
mixer's dictionary of the configuration.
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path
from typing import Any, Mapping

import torch


# ------------------------------------------------------------------------ files
def read_config(folder: str | Path) -> dict[str, Any]:
    return json.loads((Path(folder) / "config.json").read_text())


def read_weights(folder: str | Path, dtype: torch.dtype = torch.float64) -> dict[str, torch.Tensor]:
    """Parse ``model.safetensors`` by hand: 8-byte length, JSON header, raw data."""
    raw = (Path(folder) / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8: 8 + n])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + a: 8 + n + b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        out[name] = t if info["dtype"] == "I32" else t.to(dtype)
    return out


# -------------------------------------------------------------------- mechanisms
def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm of the stream: the weight is stored around zero (gain ``1 + w``)."""
    return over_rms(x, eps) * (1 + weight)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu(z: torch.Tensor) -> torch.Tensor:
    """The exact form: z times the normal distribution's cumulative probability at z."""
    return z * 0.5 * (1 + torch.erf(z / math.sqrt(2.0)))


def position_vectors(count: int, width: int, base: float = 10000.0, dtype: torch.dtype = torch.float64) -> torch.Tensor:
    """Row p: sine at the even entries, cosine at the odd ones, a frequency per pair of entries."""
    out = torch.zeros(count, width, dtype=torch.float64)
    for p in range(count):
        for c in range(width):
            angle = p * base ** (-2.0 * (c // 2) / width)
            out[p, c] = math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return out.to(dtype)


def embedding(cfg: Mapping[str, Any], w: Mapping[str, torch.Tensor], tokens: list[int]) -> torch.Tensor:
    x = w["embed"][tokens]
    return x * float(cfg["embedding"]["scale"]) + position_vectors(len(tokens), int(cfg["width"]), dtype=x.dtype)


def first_visible(i: int, chunk: int | None) -> int:
    """The first position that position i sees: the start of its chunk, counted from position 0."""
    return 0 if chunk is None else i // chunk * chunk


def attention_map(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: int | None) -> torch.Tensor:
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, dv]``: softmax attention inside chunks."""
    t, heads, _ = q.shape
    per = heads // k.shape[1]
    out = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        lo = first_visible(i, chunk)
        for a in range(heads):
            s = (k[lo: i + 1, a // per] @ q[i, a]) * scale
            e = torch.exp(s - s.max())
            out[i, a] = (e / e.sum()) @ v[lo: i + 1, a // per]
    return out


def mix_factor(w: Mapping[str, torch.Tensor], p: str, diff: float) -> torch.Tensor:
    """The factor on the second map, one number for a layer."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def chunk_of(m: Mapping[str, Any]) -> int | None:
    mask = m.get("mask")
    return None if not mask else int(mask["size"])


def combine_maps(a1: torch.Tensor, a2: torch.Tensor, factor: "torch.Tensor | float", eps: float, diff: float) -> torch.Tensor:
    return over_rms(a1 - factor * a2, eps) * (1 - diff)


def attention_mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping[str, Any], eps: float) -> torch.Tensor:
    """Two attention maps over the same values, the second subtracted with a learned factor."""
    t, heads, groups, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = over_rms((h @ w[p + "q"].T).view(t, heads, 2, d), eps) * w[p + "q.norm"]
    k = over_rms((h @ w[p + "k"].T).view(t, groups, 2, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(t, groups, dv)
    a1, a2 = (attention_map(q[:, :, n], k[:, :, n], v, float(m["scale"]), chunk_of(m)) for n in (0, 1))
    o = combine_maps(a1, a2, mix_factor(w, p, float(m["diff"])), eps, float(m["diff"]))
    return o.reshape(t, -1) @ w[p + "o"].T


def short_conv(u: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """``u [T, channels]``: every channel is the weighted sum of its last values plus a bias, the last
    tap on the current token; zeros before the start."""
    t, k = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for n in range(t):
        out[n] = bias
        for j in range(k):
            src = n - (k - 1) + j
            if src >= 0:
                out[n] += taps[:, j] * u[src]
    return out


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def state_space_scan(x: torch.Tensor, b: torch.Tensor, c: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor,
                     state: torch.Tensor | None = None) -> torch.Tensor:
    """``x [T, H, dv]``, ``b``/``c`` ``[T, G, N]``, ``dt [T, H]`` (after softplus): per head
    ``S <- exp(-exp(A) dt) S + dt b x^T``, ``y = S^T c + D x`` token by token (``state`` is changed)."""
    t, heads, dv = x.shape
    per = heads // b.shape[1]
    s = torch.zeros(heads, b.shape[-1], dv, dtype=x.dtype) if state is None else state
    y = torch.zeros_like(x)
    for n in range(t):
        for a in range(heads):
            decay = torch.exp(-torch.exp(a_log[a]) * dt[n, a])
            s[a] = decay * s[a] + dt[n, a] * torch.outer(b[n, a // per], x[n, a])
            y[n, a] = s[a].T @ c[n, a // per] + skip[a] * x[n, a]
    return y


def gate_and_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """``y``, ``z`` ``[T, inner]``: gated, then normed part by part."""
    t, inner = y.shape
    g = y * silu(z)
    return over_rms(g.view(t, parts, inner // parts), eps).reshape(t, inner) * weight


def mamba2_mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping[str, Any], eps: float) -> torch.Tensor:
    t, heads, dv, n, g = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = heads * dv
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner: 2 * inner + 2 * g * n], proj[:, 2 * inner + 2 * g * n:]
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = xbc[:, :inner], xbc[:, inner: inner + g * n], xbc[:, inner + g * n:]
    y = state_space_scan(x.reshape(t, heads, dv), b.reshape(t, g, n), c.reshape(t, g, n), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"],
                         w[p + "D"])
    return gate_and_norm(y.reshape(t, inner), z, w[p + "norm"], int(m["norm_groups"]), eps) @ w[p + "o"].T


def dense_ff(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, router: Mapping[str, Any]) -> list[list[tuple[int, float]]]:
    """Per token the chosen (output, weight) pairs: chosen by score plus correction, weighted by
    the scores alone over their sum."""
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    choice = s + w[p + "correction"]
    picks = []
    for n in range(h.shape[0]):
        chosen = sorted(range(s.shape[1]), key=lambda e: (-float(choice[n, e]), e))[: int(router["top"])]
        den = sum(float(s[n, e]) for e in chosen) + 1e-20
        picks.append([(e, float(s[n, e]) / den * float(router.get("scale", 1.0))) for e in chosen])
    return picks


def moe_ff(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, mlp: Mapping[str, Any]) -> torch.Tensor:
    real = int(mlp["router"]["experts"])
    out = torch.zeros_like(h)
    for n, chosen in enumerate(route(h, w, p, mlp["router"])):
        for e, weight in chosen:
            out[n] += weight * (h[n] if e >= real else expert(h[n: n + 1], w, f"{p}e{e}.")[0])
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


MIXERS = {"attention": attention_mixer, "mamba2": mamba2_mixer}


def layer(x: torch.Tensor, w: Mapping[str, torch.Tensor], i: int, spec: Mapping[str, Any], eps: float) -> torch.Tensor:
    p = f"l{i}."
    x = x + MIXERS[spec["type"]](layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    mlp = spec.get("mlp")
    if mlp is not None:
        h = layer_norm(x, w[p + "norm2"], eps)
        x = x + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp))
    return x


def run_order(cfg: Mapping[str, Any]) -> list[tuple[int, bool]]:
    """Layers in the order they run, each with whether a pass of the loop starts there."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop = int(loop["start"]), int(loop["stop"])
    order = [(i, False) for i in range(start)]
    for _ in range(int(loop["times"])):
        order += [(i, i == start) for i in range(start, stop)]
    return order + [(i, False) for i in range(stop, n)]


def forward(cfg: Mapping[str, Any], w: Mapping[str, torch.Tensor], tokens: list[int], streams: "list | None" = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from its first token; ``streams`` collects the
    residual stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    first = embedding(cfg, w, tokens)
    x = first
    for i, starts in run_order(cfg):
        if starts:
            x = torch.cat([x, first], dim=-1) @ w["loop.in"].T
        x = layer(x, w, i, cfg["layers"][i], eps)
        if streams is not None:
            streams.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg: Mapping[str, Any], w: Mapping[str, torch.Tensor], prompt: list[int], new_tokens: int) -> list[int]:
    """Greedy continuation, recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(new_tokens):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
