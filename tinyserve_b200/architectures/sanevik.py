"""Sanevik: a pre-norm decoder whose layers are listed one by one in ``config.json`` and of which a
stretch may run several times with the same weights. Each layer has one of two mixers and optionally a
routed mixture of experts; norms have weights stored around zero, the logits come from the embedding table.

The mixers: ``attention`` (windowed grouped-query attention with YaRN-scaled rotation of neighbouring
pairs, q and k divided by their root mean square after the rotation, a learned sink logit per head) and
``parallel`` (two mixers on the same input, summed with a constant each: windowed attention behind short
convolutions with capped scores and weights mixed across the heads; and retention, linear attention with a
rotation and a constant decay per head). The experts: the largest sigmoid scores, not normalised, each
multiplying its expert's input; a clamped gated activation. The loop: layers ``start .. stop - 1`` run
``times`` times in a row, every pass with caches and states of its own; in front of every pass a learned
vector of that pass is added to the stream, in front of every pass but the first also the embedding output.

``config.json`` keys read here: ``architecture`` = "Sanevik"; ``vocab``, ``width``; ``norm.eps``; optional
``loop`` (``start, stop, times``); ``layers``: a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``. Mixer
keys by type: ``attention``: ``heads, kv_heads, dim, vdim, scale``, ``rot`` (``dims, base``, optional ``scaling``
with ``factor, original, fast, slow``), optional ``mask.size``; ``parallel``: ``left`` (those of ``attention``
plus ``softcap`` and ``conv``), ``right`` (``heads, dim, vdim, rot, decay`` (one constant per head)),
``left_scale``, ``right_scale`` (absent = 1). ``mlp``: ``kind`` = "moe" with ``router`` (``experts, top``) and
``expert`` (``ff, limit``). Optional ``max_positions`` bounds a request's length for the engine's bookkeeping.
Every size and constant comes from these keys.

What the design fixes, passed to the parts as arguments by ``to_spec``: rotation pairs (neighbours in both
attentions, halves in the retention), which attention has a sink, unit-length q and k, a soft cap,
convolutions or mixed weights, ``dim^-1/2`` on the retention's keys and its norm and SiLU gate, the routing
rule; tensor names ``embed``, ``loop.step``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``.left.*`` / ``.right.*`` for the
two mixers side by side), ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.gate|up|down``, ``final.norm``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Mapping

from ..config.base import LayerCall, LayerSpec, ModelConfig, ModelSpec, PartSpec, UnsupportedConfigError
from ..config.registry import register_architecture

ARCHITECTURE = "Sanevik"
MIXER_TYPES = ("attention", "parallel")
DEFAULT_MAX_POSITIONS = 1 << 17
_ATTENTION_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "rot")
_RIGHT_KEYS = ("heads", "dim", "vdim", "rot", "decay")
_SCALING_KEYS = ("factor", "original", "fast", "slow")


def _need(d: Mapping[str, Any], key: str, where: str) -> Any:
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise UnsupportedConfigError(f"{where} has no {key!r}")
    return d[key]


def _rotation(m: Mapping[str, Any], pairing: str, where: str) -> PartSpec:
    rot, dim = m["rot"], int(m["dim"])
    dims, base = int(_need(rot, "dims", f"{where}.rot")), float(_need(rot, "base", f"{where}.rot"))
    if dims % 2 or not 0 < dims <= dim:
        raise UnsupportedConfigError(f"{where}: rot.dims={dims} must be even and at most {dim}")
    args: dict[str, Any] = {"head_dim": dim, "rotary_dim": dims, "theta": base, "pairing": pairing}
    scaling = rot.get("scaling")
    if scaling is not None:
        args["scaling"] = {k: float(_need(scaling, k, f"{where}.rot.scaling")) for k in _SCALING_KEYS}
        if not all(v > 0 for v in args["scaling"].values()) or not base > 1:
            raise UnsupportedConfigError(f"{where}: rot.scaling={dict(scaling)} needs positive values and a base above 1")
    return PartSpec("rope", args)


def _window(m: Mapping[str, Any], where: str) -> int | None:
    mask = m.get("mask")
    if mask is None:
        return None
    size = int(_need(mask, "size", f"{where}.mask"))
    if size <= 0:
        raise UnsupportedConfigError(f"{where}.mask: size={size} must be positive")
    return size


@dataclass(frozen=True)
class SanevikConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple[Mapping[str, Any], ...]
    loop: tuple[int, int, int] | None = None          # first layer, the layer behind the last, passes
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
            if kind not in MIXER_TYPES:
                raise UnsupportedConfigError(f"{where}: unknown mixer type {kind!r}; known: {MIXER_TYPES}")
            m = _need(layer, "mixer", where)
            if kind == "attention":
                self._check_attention(m, f"{where}.mixer")
            else:
                left, right = _need(m, "left", f"{where}.mixer"), _need(m, "right", f"{where}.mixer")
                self._check_attention(left, f"{where}.mixer.left")
                for key in ("softcap", "conv"):
                    _need(left, key, f"{where}.mixer.left")
                if not float(left["softcap"]) > 0 or int(left["conv"]) < 1:
                    raise UnsupportedConfigError(f"{where}.mixer.left: softcap must be positive and conv at least 1")
                for key in _RIGHT_KEYS:
                    _need(right, key, f"{where}.mixer.right")
                if len(right["decay"]) != int(right["heads"]):
                    raise UnsupportedConfigError(f"{where}.mixer.right: {len(right['decay'])} decay constants for {right['heads']} heads")
                _rotation(right, "half", f"{where}.mixer.right")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if _need(mlp, "kind", f"{where}.mlp") != "moe":
                raise UnsupportedConfigError(f"{where}: mlp.kind={mlp['kind']!r}: only 'moe' is implemented")
            router, expert = _need(mlp, "router", f"{where}.mlp"), _need(mlp, "expert", f"{where}.mlp")
            if not 0 < int(_need(router, "top", "router")) <= int(_need(router, "experts", "router")):
                raise UnsupportedConfigError(f"{where}: top={router['top']} of {router['experts']} experts")
            if int(_need(expert, "ff", "expert")) <= 0 or not float(_need(expert, "limit", "expert")) > 0:
                raise UnsupportedConfigError(f"{where}: expert ff={expert['ff']} and limit={expert['limit']} must be positive")

    @staticmethod
    def _check_attention(m: Mapping[str, Any], where: str) -> None:
        for key in _ATTENTION_KEYS:
            _need(m, key, where)
        if int(m["heads"]) % int(m["kv_heads"]):
            raise UnsupportedConfigError(f"{where}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
        _rotation(m, "interleaved", where)
        _window(m, where)

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "SanevikConfig":
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
            max_positions=int(d.get("max_positions", DEFAULT_MAX_POSITIONS)),
        )

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "layers": [copy.deepcopy(dict(layer)) for layer in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d

    # ------------------------------------------------------------------ the spec
    def _attention(self, m: Mapping[str, Any], prefix: str, **more: Any) -> PartSpec:
        return PartSpec("rotated_attention", {
            "prefix": prefix, "hidden_size": self.hidden_size, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
            "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "scale": float(m["scale"]), "window": _window(m, prefix),
            "norm_eps": self.norm_eps, **more})

    def _mixers(self, kind: str, m: Mapping[str, Any]) -> tuple[dict[str, PartSpec], dict[str, PartSpec], dict[str, float]]:
        """The mixer roles of a layer, their position encodings, and the block's constants for them."""
        if kind == "attention":
            return {"mixer": self._attention(m, "mix.", unit_norm=True, sink=True)}, \
                {"mixer": _rotation(m, "interleaved", "mixer")}, {}
        left, right = m["left"], m["right"]
        retention = PartSpec("retention", {
            "prefix": "mix.right.", "hidden_size": self.hidden_size, "num_heads": int(right["heads"]), "key_dim": int(right["dim"]),
            "value_dim": int(right["vdim"]), "decay": [float(x) for x in right["decay"]], "norm_eps": self.norm_eps})
        return {"mixer": self._attention(left, "mix.left.", softcap=float(left["softcap"]), talk=True, conv_taps=int(left["conv"])),
                "second_mixer": retention}, \
            {"mixer": _rotation(left, "interleaved", "left"), "second_mixer": _rotation(right, "half", "right")}, \
            {"mixer_scale": float(m.get("left_scale", 1.0)), "second_mixer_scale": float(m.get("right_scale", 1.0))}

    def _order(self) -> tuple[LayerCall, ...]:
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(i) for i in range(n))
        start, stop, times = self.loop
        calls = [LayerCall(i) for i in range(start)]
        for t in range(times):
            step = PartSpec("pass_vector", {"name": "loop.step", "hidden_size": self.hidden_size, "index": t, "count": times,
                                            "add_origin": t > 0})
            calls += [LayerCall(i, stream_input=step if i == start else None) for i in range(start, stop)]
        return tuple(calls + [LayerCall(i) for i in range(stop, n)])

    def to_spec(self) -> ModelSpec:
        h = self.hidden_size

        def norm(name: str) -> PartSpec:
            return PartSpec("rms_norm", {"name": name, "size": h, "eps": self.norm_eps, "unit_offset": True})

        layers = []
        for i, layer in enumerate(self.layers):
            mixers, positions, block_args = self._mixers(layer["type"], layer["mixer"])
            parts = {"mixer_norm": norm("norm1"), **mixers}
            mlp = layer.get("mlp")
            if mlp is not None:
                parts["feed_forward_norm"] = norm("norm2")
                parts["feed_forward"] = PartSpec("routed_experts", {
                    "prefix": "mlp.", "hidden_size": h, "num_experts": int(mlp["router"]["experts"]), "top": int(mlp["router"]["top"]),
                    "expert_size": int(mlp["expert"]["ff"]), "routing": "scored", "score": "sigmoid", "normalise": False,
                    "weight_on": "input", "activation": "clamped_swish", "limit": float(mlp["expert"]["limit"])})
            layers.append(LayerSpec(prefix=f"l{i}.", block="prenorm", parts=parts, positions=positions, block_args=block_args))
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab_size, hidden_size=h, layers=tuple(layers), order=self._order(),
            embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": self.vocab_size, "hidden_size": h}),
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"name": "embed", "tied": True, "vocab_size": self.vocab_size, "hidden_size": h}),
            max_position_embeddings=self.max_positions,
        )


register_architecture(ARCHITECTURE, SanevikConfig)
