"""Risonex: a pre-norm decoder whose layers are listed one by one in ``config.json`` and of which a stretch may run
several times with the same weights. Each layer has one of two mixers and optionally a feed-forward, dense or a routed
mixture of experts; norms have weights stored around zero, the output head is a matrix of its own.

The mixers: ``attention`` (differential attention: two maps per head over the same values, q and k RMS-normed per
head and map, no rotation, visible keys in chunks of fixed size counted from position 0) and ``mamba2`` (a matrix
state per head with one decay per head and token; short convolutions with a bias; the gate before a norm in equal
parts). The feed-forwards: ``dense`` (two products with the exact gelu between them) and ``moe`` (SwiGLU experts chosen
by softmax score plus correction, identity experts among them, and a gated shared expert). Positions enter only
through a sinusoid added to the embedding. The loop: layers ``start .. stop - 1`` run ``times`` times in a row, every
pass with caches and states of its own; in front of every pass the stream becomes ``W_in [x; x0]`` with x0 the
embedding output.

``config.json`` keys read here: ``architecture`` = "Risonex"; ``vocab``, ``width``; ``norm.eps``; ``embedding.scale`` (absent =
1); optional ``loop`` (``start, stop, times``); ``layers``: a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``. Mixer
keys by type: ``attention``: ``heads, kv_heads, dim, vdim, scale, diff``, optional ``mask.size``; ``mamba2``: ``heads, groups,
state, vdim, conv, norm_groups``. ``mlp``: ``kind`` = "dense" with ``ff``, or "moe" with ``router`` (``experts, top``, optional
``identity``, ``scale``), ``expert.ff`` and optional ``shared.ff``. Optional ``max_positions`` bounds a request's length for
the engine's bookkeeping. Every size and constant comes from these keys.

What the design fixes, passed to the parts as arguments by ``to_spec``: the sinusoid's base 10,000, which norms have
plain weights, softmax scores over all router outputs with a correction for the choice only, the shared expert's
gate, the activations; tensor names ``embed``, ``loop.in``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from ..config.base import LayerCall, LayerSpec, ModelConfig, ModelSpec, PartSpec, UnsupportedConfigError
from ..config.registry import register_architecture

ARCHITECTURE = "Risonex"
DEFAULT_MAX_POSITIONS = 1 << 17
_MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale", "diff"),
               "mamba2": ("heads", "groups", "state", "vdim", "conv", "norm_groups")}


def _need(d: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise UnsupportedConfigError(f"{where} has no {key!r}")
    return d[key]


def _chunk(m: Mapping[str, Any], where: str) -> int | None:
    mask = m.get("mask")
    if mask is None:
        return None
    size = int(_need(mask, "size", f"{where}.mask"))
    if size <= 0:
        raise UnsupportedConfigError(f"{where}.mask: size={size} must be positive")
    return size


@dataclass(frozen=True)
class RisonexConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple[Mapping[str, Any], ...]
    loop: tuple[int, int, int] | None = None          # first layer, the layer behind the last, passes
    embedding_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    architecture = ARCHITECTURE

    def __post_init__(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0 or not self.norm_eps > 0:
            raise UnsupportedConfigError("vocab, width and norm.eps must be positive")
        if not self.layers:
            raise UnsupportedConfigError("layers is empty")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise UnsupportedConfigError(f"loop start={start} stop={stop} times={times} does not fit {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in _MIXER_KEYS:
                raise UnsupportedConfigError(f"{where}: unknown mixer type {kind!r}; known: {tuple(_MIXER_KEYS)}")
            m = _need(layer, "mixer", where)
            for key in _MIXER_KEYS[kind]:
                _need(m, key, f"{where}.mixer")
            if kind == "attention":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise UnsupportedConfigError(f"{where}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
                _chunk(m, f"{where}.mixer")
            else:
                if int(m["heads"]) % int(m["groups"]):
                    raise UnsupportedConfigError(f"{where}: heads={m['heads']} is not a multiple of groups={m['groups']}")
                if int(m["heads"]) * int(m["vdim"]) % int(m["norm_groups"]):
                    raise UnsupportedConfigError(f"{where}: norm_groups={m['norm_groups']} does not divide {m['heads']} x {m['vdim']} columns")
                if int(m["conv"]) < 1:
                    raise UnsupportedConfigError(f"{where}: conv={m['conv']} must be at least 1")
            mlp = layer.get("mlp")
            if mlp is not None:
                self._check_mlp(mlp, f"{where}.mlp")

    @staticmethod
    def _check_mlp(mlp: Mapping[str, Any], where: str) -> None:
        kind = _need(mlp, "kind", where)
        if kind == "dense":
            if int(_need(mlp, "ff", where)) <= 0:
                raise UnsupportedConfigError(f"{where}: ff={mlp['ff']} must be positive")
            return
        if kind != "moe":
            raise UnsupportedConfigError(f"{where}: mlp.kind={kind!r}: 'dense' and 'moe' are implemented")
        router = _need(mlp, "router", where)
        experts, top, identity = int(_need(router, "experts", "router")), int(_need(router, "top", "router")), int(router.get("identity", 0))
        if experts <= 0 or identity < 0 or not 0 < top <= experts + identity:
            raise UnsupportedConfigError(f"{where}: top={top} of {experts} experts and {identity} identity experts")
        for part in ("expert", "shared"):
            if (part == "expert" or mlp.get(part) is not None) and int(_need(_need(mlp, part, where), "ff", f"{where}.{part}")) <= 0:
                raise UnsupportedConfigError(f"{where}.{part}: ff={mlp[part]['ff']} must be positive")

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RisonexConfig":
        name = d.get("architecture") or (d.get("architectures") or [None])[0]
        if name != ARCHITECTURE:
            raise UnsupportedConfigError(f"expected {ARCHITECTURE}, got {name!r}")
        loop = d.get("loop")
        return cls(
            vocab_size=int(_need(d, "vocab", "config.json")),
            hidden_size=int(_need(d, "width", "config.json")),
            norm_eps=float(_need(_need(d, "norm", "config.json"), "eps", "norm")),
            layers=tuple(copy.deepcopy(dict(layer)) for layer in _need(d, "layers", "config.json")),
            loop=None if loop is None else tuple(int(_need(loop, k, "loop")) for k in ("start", "stop", "times")),
            embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
            max_positions=int(d.get("max_positions", DEFAULT_MAX_POSITIONS)),
        )

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                             "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                             "layers": [copy.deepcopy(dict(layer)) for layer in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d

    # ------------------------------------------------------------------ the spec
    def _mixer(self, kind: str, m: Mapping[str, Any]) -> PartSpec:
        if kind == "attention":
            return PartSpec("differential_attention", {
                "prefix": "mix.", "hidden_size": self.hidden_size, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
                "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "scale": float(m["scale"]), "diff": float(m["diff"]),
                "norm_eps": self.norm_eps, "chunk": _chunk(m, "mixer")})
        return PartSpec("state_space", {
            "prefix": "mix.", "hidden_size": self.hidden_size, "num_heads": int(m["heads"]), "num_groups": int(m["groups"]),
            "state_dim": int(m["state"]), "value_dim": int(m["vdim"]), "conv_taps": int(m["conv"]),
            "norm_parts": int(m["norm_groups"]), "norm_eps": self.norm_eps})

    def _feed_forward(self, mlp: Mapping[str, Any]) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("plain_mlp", {"prefix": "mlp.", "hidden_size": self.hidden_size, "intermediate_size": int(mlp["ff"]),
                                          "activation": "gelu"})
        router, shared = mlp["router"], mlp.get("shared")
        return PartSpec("routed_experts", {
            "prefix": "mlp.", "hidden_size": self.hidden_size, "num_experts": int(router["experts"]), "top": int(router["top"]),
            "expert_size": int(mlp["expert"]["ff"]), "shared_size": None if shared is None else int(shared["ff"]),
            "routing": "scored", "correction": True, "route_scale": float(router.get("scale", 1.0)),
            "identity": int(router.get("identity", 0)), "shared_gate": shared is not None})

    def _order(self) -> tuple[LayerCall, ...]:
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(i) for i in range(n))
        start, stop, times = self.loop
        enter = PartSpec("pass_projection", {"name": "loop.in", "hidden_size": self.hidden_size})
        one_pass = [LayerCall(i, stream_input=enter if i == start else None) for i in range(start, stop)]
        return tuple([LayerCall(i) for i in range(start)] + one_pass * times + [LayerCall(i) for i in range(stop, n)])

    def to_spec(self) -> ModelSpec:
        h = self.hidden_size

        def norm(name: str) -> PartSpec:
            return PartSpec("rms_norm", {"name": name, "size": h, "eps": self.norm_eps, "unit_offset": True})

        layers = []
        for i, layer in enumerate(self.layers):
            parts = {"mixer_norm": norm("norm1"), "mixer": self._mixer(layer["type"], layer["mixer"])}
            if layer.get("mlp") is not None:
                parts["feed_forward_norm"] = norm("norm2")
                parts["feed_forward"] = self._feed_forward(layer["mlp"])
            layers.append(LayerSpec(prefix=f"l{i}.", block="prenorm", parts=parts))
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab_size, hidden_size=h, layers=tuple(layers), order=self._order(),
            embedding=PartSpec("sinusoidal_embedding", {"name": "embed", "vocab_size": self.vocab_size, "hidden_size": h,
                                                        "scale": self.embedding_scale, "base": 10000.0}),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"name": "head", "tied": False, "vocab_size": self.vocab_size, "hidden_size": h}),
            max_position_embeddings=self.max_positions,
        )


register_architecture(ARCHITECTURE, RisonexConfig)
