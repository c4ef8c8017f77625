"""Lasupel: typed configuration and its description as parts.

A decoder whose config.json lists its layers one by one.  The embedding is multiplied by ``embedding.scale``; a layer
is x <- x + norm1(mixer(x)), then, where it has a feed-forward, x <- x + norm2(ff(x)): the sublayers read the stream
itself and only what they give is normed (RMS norms with a weight).  The stream x is float32 also in the bfloat16
path.  Three mixers:

``attention``  grouped-query attention over a sliding window (``mask.size``; none: all keys); the first ``rot.dims``
               dimensions of q and k heads turn as paired halves, q and k heads are divided by their root mean
               square, and the softmax has one more term of score 0 in its denominator.  A layer with ``kv_from: j``
               has no keys and values of its own: it reads those that layer j caches, through its own window.
``rglru``      a linear recurrent unit of ``width`` channels behind a short convolution (``conv`` taps), its gates
               square matrices over ``blocks`` parts of the channels, beside a GELU branch that multiplies it.
``delta``      the gated delta rule: ``heads`` states [dim, vdim] whose q and k come from ``kv_heads`` heads, all of
               q, k and v through short convolutions with SiLU.

The feed-forward is dense, down(silu(gate h) * (up h)), or a mixture of gated experts with limits, routed by a softmax
over all experts with groups, or absent.  All of it maps onto parts of the package with these numbers as parameters;
nothing here computes.

Checkpoint names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.{q,k,v,o}`` (``{q,o}`` with ``kv_from``),
``l<i>.mix.{y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,lam,o}``, ``l<i>.mix.{q,q.conv,k,k.conv,v,v.conv,b,a,A_log,dt_bias,
g,norm,o}``, ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down}``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from ..config.registry import ConfigError, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunStep

MIXER_TYPES = ("attention", "rglru", "delta")
# the experts' activation is g * sigmoid(EXPERT_ALPHA * g) * (u + 1)
EXPERT_ALPHA = 1.702
# the score of the softmax's extra term
SINK_SCORE = 0.0
# log a = -DECAY_POWER * r * softplus(lam) in the linear recurrent unit
DECAY_POWER = 8.0
# inside the root of the delta rule's unit vectors
UNIT_EPS = 1e-6
# positions enter through computed angles and distances, none tabulated: the engine's own max_model_len bounds a request
UNBOUNDED_POSITIONS = 1 << 20


def _positive_int(name: str, value: Any) -> int:
    if type(value) is not int or value <= 0:
        raise ConfigError(f"{name} must be a positive integer, got {value!r}")
    return value


def _number(name: str, value: Any) -> float:
    if type(value) not in (int, float):
        raise ConfigError(f"{name} must be a number, got {value!r}")
    return float(value)


def _need(where: str, data: Any, keys) -> Mapping[str, Any]:
    if not isinstance(data, Mapping):
        raise ConfigError(f"{where} must be an object")
    missing = [key for key in keys if key not in data]
    if missing:
        raise ConfigError(f"{where} lacks " + ", ".join(missing))
    return data


@dataclass(frozen=True)
class LasupelFeedForward:
    kind: str                              # "dense" or "moe"
    ff: int                                # dense: the inner size; moe: an expert's
    limit: float = 0.0                     # moe from here on
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1

    def __post_init__(self) -> None:
        if self.kind not in ("dense", "moe"):
            raise ConfigError(f"mlp.kind is 'dense' or 'moe', not {self.kind!r}")
        _positive_int("mlp.ff", self.ff)
        if self.kind == "moe":
            if not self.limit > 0:
                raise ConfigError("mlp.expert.limit must be positive")
            _positive_int("mlp.router.experts", self.experts)
            _positive_int("mlp.router.top", self.top)
            _positive_int("mlp.router.groups.count", self.groups)
            _positive_int("mlp.router.groups.keep", self.keep)
            if self.experts % self.groups or self.keep > self.groups:
                raise ConfigError("mlp.router.groups must divide the experts, and keep at most all groups")
            if self.top > self.experts // self.groups * self.keep:
                raise ConfigError("mlp.router.top must not exceed the experts of the groups that are kept")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "LasupelFeedForward":
        data = _need(where, data, ("kind",))
        if data["kind"] == "dense":
            return cls(kind="dense", ff=_need(where, data, ("ff",))["ff"])
        if data["kind"] != "moe":
            raise ConfigError(f"{where}.kind is 'dense' or 'moe', not {data['kind']!r}")
        data = _need(where, data, ("expert", "router"))
        expert = _need(f"{where}.expert", data["expert"], ("ff", "limit"))
        router = _need(f"{where}.router", data["router"], ("experts", "top"))
        groups = router.get("groups")
        count = keep = 1
        if groups is not None:
            groups = _need(f"{where}.router.groups", groups, ("count", "keep"))
            count, keep = groups["count"], groups["keep"]
        return cls(kind="moe", ff=expert["ff"], limit=_number("mlp.expert.limit", expert["limit"]),
                   experts=router["experts"], top=router["top"], groups=count, keep=keep)

    def to_json(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        return {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep},
                           "top": self.top}}


@dataclass(frozen=True)
class LasupelAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None = None              # None: all keys
    rot_dims: int = 0                      # 0: no rotation
    rot_base: float = 0.0
    kv_from: int | None = None             # the layer whose keys and values are read

    type = "attention"

    def __post_init__(self) -> None:
        for name in ("heads", "kv_heads", "dim", "vdim"):
            _positive_int(f"mixer.{name}", getattr(self, name))
        if self.heads % self.kv_heads:
            raise ConfigError("mixer.heads must be a multiple of mixer.kv_heads")
        if self.window is not None:
            _positive_int("mixer.mask.size", self.window)
        if type(self.rot_dims) is not int or self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ConfigError("mixer.rot.dims must be even and at most mixer.dim")
        if self.rot_dims and not self.rot_base > 0:
            raise ConfigError("mixer.rot.base must be positive")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "LasupelAttention":
        data = _need(where, data, ("heads", "kv_heads", "dim", "vdim", "scale"))
        rot, mask = data.get("rot"), data.get("mask")
        rotation = {}
        if rot is not None:
            rot = _need(f"{where}.rot", rot, ("dims", "base"))
            rotation = {"rot_dims": rot["dims"], "rot_base": _number("mixer.rot.base", rot["base"])}
        return cls(heads=data["heads"], kv_heads=data["kv_heads"], dim=data["dim"], vdim=data["vdim"],
                   scale=_number("mixer.scale", data["scale"]),
                   window=None if mask is None else _need(f"{where}.mask", mask, ("size",))["size"],
                   kv_from=data.get("kv_from"), **rotation)

    def to_json(self) -> dict[str, Any]:
        data: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                                "vdim": self.vdim}
        if self.kv_from is not None:
            data["kv_from"] = self.kv_from
        if self.window is not None:
            data["mask"] = {"size": self.window}
        if self.rot_dims:
            data["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return data


@dataclass(frozen=True)
class LasupelRecurrentUnit:
    width: int
    blocks: int
    conv: int

    type = "rglru"

    def __post_init__(self) -> None:
        for name in ("width", "blocks", "conv"):
            _positive_int(f"mixer.{name}", getattr(self, name))
        if self.width % self.blocks:
            raise ConfigError("mixer.blocks must divide mixer.width")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "LasupelRecurrentUnit":
        keys = ("width", "blocks", "conv")
        data = _need(where, data, keys)
        return cls(**{key: data[key] for key in keys})

    def to_json(self) -> dict[str, Any]:
        return {"blocks": self.blocks, "conv": self.conv, "width": self.width}


@dataclass(frozen=True)
class LasupelDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    type = "delta"

    def __post_init__(self) -> None:
        for name in ("heads", "kv_heads", "dim", "vdim", "conv"):
            _positive_int(f"mixer.{name}", getattr(self, name))
        if self.heads % self.kv_heads:
            raise ConfigError("mixer.heads must be a multiple of mixer.kv_heads")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "LasupelDelta":
        keys = ("heads", "kv_heads", "dim", "vdim", "conv")
        data = _need(where, data, keys)
        return cls(**{key: data[key] for key in keys})

    def to_json(self) -> dict[str, Any]:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


MIXERS = {mixer.type: mixer for mixer in (LasupelAttention, LasupelRecurrentUnit, LasupelDelta)}


@dataclass(frozen=True)
class LasupelLayer:
    mixer: LasupelAttention | LasupelRecurrentUnit | LasupelDelta
    mlp: LasupelFeedForward | None = None

    @property
    def type(self) -> str:
        return self.mixer.type

    @classmethod
    def from_json(cls, index: int, data: Any) -> "LasupelLayer":
        where = f"layers[{index}]"
        data = _need(where, data, ("type", "mixer"))
        if data["type"] not in MIXERS:
            raise ConfigError(f"{where}.type is one of {', '.join(MIXER_TYPES)}, not {data['type']!r}")
        mlp = data.get("mlp")
        return cls(mixer=MIXERS[data["type"]].from_json(f"{where}.mixer", data["mixer"]),
                   mlp=None if mlp is None else LasupelFeedForward.from_json(f"{where}.mlp", mlp))

    def to_json(self) -> dict[str, Any]:
        return {"mixer": self.mixer.to_json(), "mlp": None if self.mlp is None else self.mlp.to_json(),
                "type": self.type}


@dataclass(frozen=True)
class LasupelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[LasupelLayer, ...]
    embedding_scale: float = 1.0
    eos_token_ids: tuple[int, ...] = ()

    architecture = "Lasupel"

    def __post_init__(self) -> None:
        _positive_int("vocab", self.vocab)
        _positive_int("width", self.width)
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        for index, layer in enumerate(self.layers):
            source = getattr(layer.mixer, "kv_from", None)
            if source is None:
                continue
            if type(source) is not int or not 0 <= source < index:
                raise ConfigError(f"layers[{index}].mixer.kv_from must name an earlier layer")
            owner, reader = self.layers[source].mixer, layer.mixer
            if owner.type != "attention" or owner.kv_from is not None:
                raise ConfigError(f"layers[{index}].mixer.kv_from names a layer without keys and values of its own")
            if (owner.kv_heads, owner.dim, owner.vdim) != (reader.kv_heads, reader.dim, reader.vdim):
                raise ConfigError(f"layers[{index}] reads keys and values of other sizes than its own")

    @classmethod
    def from_json(cls, data: Mapping[str, Any]) -> "LasupelConfig":
        data = _need("config.json", data, ("vocab", "width", "norm", "layers"))
        norm = _need("config.json 'norm'", data["norm"], ("eps",))
        if not isinstance(data["layers"], list):
            raise ConfigError("config.json 'layers' must be a list")
        embedding = _need("embedding", data.get("embedding") or {}, ())
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if type(eos) is int else tuple(eos)
        return cls(vocab=data["vocab"], width=data["width"], norm_eps=_number("norm.eps", norm["eps"]),
                   layers=tuple(LasupelLayer.from_json(i, layer) for i, layer in enumerate(data["layers"])),
                   embedding_scale=_number("embedding.scale", embedding.get("scale", 1.0)), eos_token_ids=eos_ids)

    def to_json(self) -> dict[str, Any]:
        data: dict[str, Any] = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                                "layers": [layer.to_json() for layer in self.layers],
                                "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.eos_token_ids:
            data["eos_token_id"] = list(self.eos_token_ids)
        return data

    # ------------------------------------------------------------------ spec
    def _mixer_spec(self, mixer) -> PartSpec:
        if mixer.type == "rglru":
            return PartSpec("linear_recurrent_unit", {
                "hidden_size": self.width, "channels": mixer.width, "blocks": mixer.blocks, "taps": mixer.conv,
                "decay_power": DECAY_POWER, "activation": "gelu_tanh", "float32_output": True})
        if mixer.type == "delta":
            return PartSpec("gated_delta_rule", {
                "hidden_size": self.width, "num_heads": mixer.heads, "num_key_heads": mixer.kv_heads,
                "key_dim": mixer.dim, "value_dim": mixer.vdim, "taps": mixer.conv,
                "query_scale": float(mixer.dim) ** -0.5, "unit_eps": UNIT_EPS, "out_norm": "weight",
                "eps": self.norm_eps, "gate": "silu", "float32_output": True})
        position = None
        if mixer.rot_dims:
            position = PartSpec("rope_half_split_computed", {"dims": mixer.rot_dims, "base": mixer.rot_base})
        # a rotation moves no length: the unit norm over a head is the same before it and behind it
        return PartSpec("windowed_attention", {
            "hidden_size": self.width, "num_heads": mixer.heads, "num_kv_heads": mixer.kv_heads,
            "key_dim": mixer.dim, "value_dim": mixer.vdim, "scale": mixer.scale, "window": mixer.window,
            "qk_norm": "unit", "qk_norm_eps": self.norm_eps, "position": position, "sink": SINK_SCORE,
            "reads_other_cache": mixer.kv_from is not None, "float32_output": True})

    def _feed_forward_spec(self, mlp: LasupelFeedForward | None) -> PartSpec | None:
        if mlp is None:
            return None
        if mlp.kind == "dense":
            return PartSpec("gated_mlp", {
                "hidden_size": self.width, "intermediate_size": mlp.ff, "activation": "silu",
                "float32_output": True, "names": {"gate": "gate", "up": "up", "down": "down"}})
        return PartSpec("softmax_routed_experts", {
            "hidden_size": self.width, "experts": mlp.experts, "top": mlp.top, "ff": mlp.ff, "limit": mlp.limit,
            "alpha": EXPERT_ALPHA, "groups": mlp.groups, "keep": mlp.keep, "float32_output": True})

    def to_spec(self) -> ModelSpec:
        norm = PartSpec("rms_norm_stream32", {"width": self.width, "eps": self.norm_eps})
        block = PartSpec("output_norm_residual", {"mixer_norm_name": "norm1", "feed_forward_norm_name": "norm2",
                                                  "mixer_name": "mix", "feed_forward_name": "mlp"})
        layers = tuple(LayerSpec(prefix=f"l{index}", block=block, mixer=self._mixer_spec(layer.mixer),
                                 feed_forward=self._feed_forward_spec(layer.mlp), norm=norm)
                       for index, layer in enumerate(self.layers))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=UNBOUNDED_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "width": self.width, "name": "embed",
                                                   "stream_scale": self.embedding_scale}),
            layers=layers,
            order=tuple(RunStep(index, getattr(layer.mixer, "kv_from", None)) for index, layer in enumerate(self.layers)),
            final_norm=norm.with_params(name="final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "width": self.width, "tied_to": None, "name": "head"}),
            eos_token_ids=self.eos_token_ids)


register_architecture(LasupelConfig.architecture, LasupelConfig)
