"""A plain, slow implementation of the Sanevik decoder, one function per mechanism, written from
the design's equations and sharing no code with the product path. Everything runs token by token or
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
def rms_norm(x: torch.Tensor, weight: torch.Tensor | None, eps: float) -> torch.Tensor:
    """Divided by the root mean square; a weight is stored around zero (gain ``1 + w``)."""
    y = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * (1 + weight)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def frequencies(rot: Mapping[str, Any]) -> tuple[list[float], float]:
    """The angle per position of every pair, and the factor on cos and sin (1 without scaling).
    With scaling (YaRN) a pair's frequency moves from itself to itself over ``factor`` along a
    ramp between the pairs that turn ``fast`` and ``slow`` times over ``original`` positions."""
    dims, base = int(rot["dims"]), float(rot["base"])
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return freq, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def pair_that_turns(times: float) -> float:
        return dims * math.log(original / (2 * math.pi * times)) / (2 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(s["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(s["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, rot: Mapping[str, Any], pairing: str, first_position: int = 0) -> torch.Tensor:
    """``x [T, heads, d]``: pairs among the first ``dims`` elements of every head turn by
    position times frequency; pairs are neighbours ("interleaved") or ``i, i + dims / 2`` ("half")."""
    dims = int(rot["dims"])
    freq, mult = frequencies(rot)
    out = x.clone()
    for n in range(x.shape[0]):
        for i, f in enumerate(freq):
            a = (first_position + n) * f
            c, s = math.cos(a) * mult, math.sin(a) * mult
            iu, iv = (2 * i, 2 * i + 1) if pairing == "interleaved" else (i, i + dims // 2)
            u, v = x[n, :, iu], x[n, :, iv]
            out[n, :, iu] = u * c - v * s
            out[n, :, iv] = v * c + u * s
    return out


def short_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """``u [T, channels]``: every channel is the weighted sum of its last values, the last tap on
    the current token; zeros before the start."""
    t, k = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for n in range(t):
        for j in range(k):
            src = n - (k - 1) + j
            if src >= 0:
                out[n] += taps[:, j] * u[src]
    return out


def softmax_with_sink(scores: torch.Tensor, sink: float | None) -> torch.Tensor:
    """Weights of one query over its visible keys; with a sink the denominator has the extra
    term ``exp(sink)``, to which no value belongs."""
    top = float(scores.max()) if sink is None else max(float(scores.max()), float(sink))
    e = torch.exp(scores - top)
    den = e.sum() + (0.0 if sink is None else math.exp(float(sink) - top))
    return e / den


def head_weights(q: torch.Tensor, k: torch.Tensor, i: int, scale: float, window: int | None, softcap: float | None,
                 sink: float | None) -> tuple[torch.Tensor, int]:
    """One head's weights of query i over the keys it sees, and the first of them."""
    lo = 0 if window is None else max(0, i - window + 1)
    s = (k[lo: i + 1] @ q[i]) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    return softmax_with_sink(s, sink), lo


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int | None,
              softcap: float | None = None, sinks: "list[float] | None" = None, talk: torch.Tensor | None = None) -> torch.Tensor:
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, dv]``; ``talk [H, H]`` mixes the heads' weights
    before each head applies its own to the values of its key/value head."""
    t, heads, _ = q.shape
    per = heads // k.shape[1]
    out = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        rows = []
        for a in range(heads):
            p, lo = head_weights(q[:, a], k[:, a // per], i, scale, window, softcap, None if sinks is None else sinks[a])
            rows.append(p)
        weights = torch.stack(rows)
        if talk is not None:
            weights = talk @ weights
        for a in range(heads):
            out[i, a] = weights[a] @ v[lo: i + 1, a // per]
    return out


def window_of(m: Mapping[str, Any]) -> int | None:
    mask = m.get("mask")
    return None if not mask else int(mask["size"])


def attention_mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping[str, Any], eps: float) -> torch.Tensor:
    """Grouped-query attention over a window, with q and k divided by their root mean square after
    the rotation and a learned sink per head."""
    t, heads, groups, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate((h @ w[p + "q"].T).view(t, heads, d), m["rot"], "interleaved")
    k = rotate((h @ w[p + "k"].T).view(t, groups, d), m["rot"], "interleaved")
    v = (h @ w[p + "v"].T).view(t, groups, dv)
    o = attention(rms_norm(q, None, eps), rms_norm(k, None, eps), v, float(m["scale"]), window_of(m),
                  sinks=[float(x) for x in w[p + "sink"]])
    return o.reshape(t, -1) @ w[p + "o"].T


def talking_mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping[str, Any]) -> torch.Tensor:
    """Windowed attention behind short convolutions, with capped scores and weights that are mixed
    across the heads after the softmax."""
    t, heads, groups, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (short_conv(h @ w[p + n].T, w[p + n + ".conv"]) for n in ("q", "k", "v"))
    q = rotate(q.view(t, heads, d), m["rot"], "interleaved")
    k = rotate(k.view(t, groups, d), m["rot"], "interleaved")
    o = attention(q, k, v.view(t, groups, dv), float(m["scale"]), window_of(m), softcap=float(m["softcap"]), talk=w[p + "talk"])
    return o.reshape(t, -1) @ w[p + "o"].T


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: "list[float]",
              state: torch.Tensor | None = None) -> torch.Tensor:
    """``S <- decay S + k v^T``, ``o = S^T q`` per head, token by token (``state`` is changed)."""
    t, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[-1], dtype=q.dtype) if state is None else state
    o = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for n in range(t):
        for a in range(heads):
            s[a] = decay[a] * s[a] + torch.outer(k[n, a], v[n, a])
            o[n, a] = s[a].T @ q[n, a]
    return o


def retention_mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping[str, Any], eps: float) -> torch.Tensor:
    t, heads, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate((h @ w[p + "q"].T).view(t, heads, d), m["rot"], "half")
    k = rotate((h @ w[p + "k"].T).view(t, heads, d), m["rot"], "half") * d ** -0.5
    v = (h @ w[p + "v"].T).view(t, heads, dv)
    o = rms_norm(retention(q, k, v, [float(x) for x in m["decay"]]), None, eps)
    return (o.reshape(t, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, spec: Mapping[str, Any], eps: float) -> torch.Tensor:
    m = spec["mixer"]
    if spec["type"] == "attention":
        return attention_mixer(h, w, p, m, eps)
    return (float(m["left_scale"]) * talking_mixer(h, w, p + "left.", m["left"])
            + float(m["right_scale"]) * retention_mixer(h, w, p + "right.", m["right"], eps))


def expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, top: int) -> list[list[tuple[int, float]]]:
    """Per token the chosen (expert, weight) pairs: the largest sigmoid scores, as they are."""
    z = h @ w[p + "router"].T
    s = torch.sigmoid(z)
    picks = []
    for n in range(h.shape[0]):
        chosen = sorted(range(z.shape[1]), key=lambda e: (-float(z[n, e]), e))[:top]
        picks.append([(e, float(s[n, e])) for e in chosen])
    return picks


def moe_ff(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, mlp: Mapping[str, Any]) -> torch.Tensor:
    """Every chosen expert runs on the token's input times its weight."""
    out = torch.zeros_like(h)
    for n, chosen in enumerate(route(h, w, p, int(mlp["router"]["top"]))):
        for e, weight in chosen:
            out[n] += expert(weight * h[n: n + 1], w, f"{p}e{e}.", float(mlp["expert"]["limit"]))[0]
    return out


def layer(x: torch.Tensor, w: Mapping[str, torch.Tensor], i: int, spec: Mapping[str, Any], eps: float) -> torch.Tensor:
    p = f"l{i}."
    x = x + mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec, eps)
    if spec.get("mlp") is not None:
        x = x + moe_ff(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", spec["mlp"])
    return x


def run_order(cfg: Mapping[str, Any]) -> list[tuple[int, int | None]]:
    """Layers in the order they run, each with the number of the loop's pass that starts there."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = int(loop["start"]), int(loop["stop"])
    order: list[tuple[int, int | None]] = [(i, None) for i in range(start)]
    for t in range(int(loop["times"])):
        order += [(i, t if i == start else None) for i in range(start, stop)]
    return order + [(i, None) for i in range(stop, n)]


def forward(cfg: Mapping[str, Any], w: Mapping[str, torch.Tensor], tokens: list[int], streams: "list | None" = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from its first token; ``streams`` collects the
    residual stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    first = w["embed"][tokens]
    x = first
    for i, starts in run_order(cfg):
        if starts is not None:
            if starts > 0:
                x = x + first
            x = x + w["loop.step"][starts]
        x = layer(x, w, i, cfg["layers"][i], eps)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg: Mapping[str, Any], w: Mapping[str, torch.Tensor], prompt: list[int], new_tokens: int) -> list[int]:
    """Greedy continuation, recomputing the whole sequence for every token."""
    toks = list(prompt)
    for _ in range(new_tokens):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
