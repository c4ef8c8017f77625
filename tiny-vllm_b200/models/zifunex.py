"""Zifunex: typed configuration and its description as parts.

A decoder whose config.json lists its layers one by one, over a residual of several streams: ``streams`` copies
of the embedding, which every sublayer reads through a stored combination and writes back through a stored
mixing matrix (hyper-connections).  A layer is pre-norm, mixer then, where it has one, feed-forward; the norms
are layer norms with weight and bias and the streams are float32 also in the bfloat16 path.  The embedding of a
token is the sum of its own row and of a row chosen by a hash of the token before it and itself.  Two mixers:

``parallel``  two mixers side by side on the same input: grouped-query attention (biases on every projection,
              the first ``rot.dims`` dimensions of a head turned as paired halves, capped scores) and a
              selective scan (Mamba: a short causal convolution, then a state a channel whose step size, input
              and output directions come from the token); the result is half the sum of the two outputs, each
              RMS-normed with a weight of its own
``gla``       gated linear attention: a float32 state a head that decays by sigmoid(z)^(1 / tau) a key
              channel, z from a two-step projection; every head's output is RMS-normed with one weight for all
              heads and gated by silu(W_g x)

The feed-forward is a dense gated one with the tanh form of GELU.  ``loop`` runs a stretch of layers several
times with the same weights; every pass has a cache and states of its own.  All of it maps onto parts of the
package with these numbers as parameters; nothing here computes.

Checkpoint names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.norm1.b``, ``l<i>.norm2``, ``l<i>.norm2.b``,
``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.{in,out,mix}``, ``l<i>.mix.left.{q,k,v,o}`` and their ``.b``,
``l<i>.mix.left.out``, ``l<i>.mix.right.{in,conv,conv.b,x,dt,dt.b,A_log,D,o}``, ``l<i>.mix.right.out``, or
``l<i>.mix.{q,k,v,g,o,norm,a1,a2,a2.b}``, ``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``final.norm.b``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from ..config.registry import ConfigError, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunStep

MIXER_TYPES = ("parallel", "gla")
# positions enter through computed angles, none tabulated: the engine's own max_model_len bounds a request
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
class ZifunexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None = None
    rot_dims: int = 0                  # 0: positions do not enter the scores
    rot_base: float = 10000.0

    def __post_init__(self) -> None:
        for name in ("heads", "kv_heads", "dim", "vdim"):
            _positive_int(f"mixer.left.{name}", getattr(self, name))
        if self.heads % self.kv_heads:
            raise ConfigError("mixer.left.heads must be a multiple of mixer.left.kv_heads")
        if type(self.rot_dims) is not int or not 0 <= self.rot_dims <= self.dim or self.rot_dims % 2:
            raise ConfigError("mixer.left.rot.dims must be an even integer of at most mixer.left.dim")
        if not self.rot_base > 0:
            raise ConfigError("mixer.left.rot.base must be positive")
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError("mixer.left.softcap must be positive")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "ZifunexAttention":
        data = _need(where, data, ("heads", "kv_heads", "dim", "vdim", "scale"))
        softcap = data.get("softcap")
        more = {}
        if data.get("rot") is not None:
            rot = _need(f"{where}.rot", data["rot"], ("dims", "base"))
            more = {"rot_dims": rot["dims"], "rot_base": _number(f"{where}.rot.base", rot["base"])}
        return cls(heads=data["heads"], kv_heads=data["kv_heads"], dim=data["dim"], vdim=data["vdim"],
                   scale=_number(f"{where}.scale", data["scale"]),
                   softcap=None if softcap is None else _number(f"{where}.softcap", softcap), **more)

    def to_json(self) -> dict[str, Any]:
        data: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads,
                                "scale": self.scale, "vdim": self.vdim}
        if self.rot_dims:
            data["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.softcap is not None:
            data["softcap"] = self.softcap
        return data


@dataclass(frozen=True)
class ZifunexScan:
    inner: int
    state: int
    dt_rank: int
    conv: int

    def __post_init__(self) -> None:
        for name in ("inner", "state", "dt_rank", "conv"):
            _positive_int(f"mixer.right.{name}", getattr(self, name))

    @classmethod
    def from_json(cls, where: str, data: Any) -> "ZifunexScan":
        keys = ("inner", "state", "dt_rank", "conv")
        data = _need(where, data, keys)
        return cls(**{key: data[key] for key in keys})

    def to_json(self) -> dict[str, Any]:
        return {"conv": self.conv, "dt_rank": self.dt_rank, "inner": self.inner, "state": self.state}


@dataclass(frozen=True)
class ZifunexLinearAttention:
    heads: int
    dim: int
    vdim: int
    tau: float

    def __post_init__(self) -> None:
        for name in ("heads", "dim", "vdim"):
            _positive_int(f"mixer.{name}", getattr(self, name))
        if not self.tau > 0:
            raise ConfigError("mixer.tau must be positive")

    @classmethod
    def from_json(cls, where: str, data: Any) -> "ZifunexLinearAttention":
        data = _need(where, data, ("heads", "dim", "vdim", "tau"))
        return cls(heads=data["heads"], dim=data["dim"], vdim=data["vdim"], tau=_number(f"{where}.tau", data["tau"]))

    def to_json(self) -> dict[str, Any]:
        return {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}


@dataclass(frozen=True)
class ZifunexLayer:
    """A layer has ``left`` and ``right`` (``parallel``) or ``linear`` (``gla``)."""

    left: ZifunexAttention | None = None
    right: ZifunexScan | None = None
    linear: ZifunexLinearAttention | None = None
    ff: int | None = None              # None: no feed-forward

    def __post_init__(self) -> None:
        if (self.left is None) != (self.right is None) or (self.left is None) == (self.linear is None):
            raise ConfigError("a layer has either two mixers side by side or gated linear attention")
        if self.ff is not None:
            _positive_int("mlp.ff", self.ff)

    @property
    def type(self) -> str:
        return "gla" if self.linear is not None else "parallel"

    @classmethod
    def from_json(cls, index: int, data: Any) -> "ZifunexLayer":
        where = f"layers[{index}]"
        data = _need(where, data, ("type", "mixer"))
        mlp, ff = data.get("mlp"), None
        if mlp is not None:
            mlp = _need(f"{where}.mlp", mlp, ("kind", "ff"))
            if mlp["kind"] != "dense":
                raise ConfigError(f"{where}.mlp.kind must be 'dense', not {mlp['kind']!r}")
            ff = mlp["ff"]
        if data["type"] == "gla":
            return cls(linear=ZifunexLinearAttention.from_json(f"{where}.mixer", data["mixer"]), ff=ff)
        if data["type"] != "parallel":
            raise ConfigError(f"{where}.type is one of {', '.join(MIXER_TYPES)}, not {data['type']!r}")
        mixer = _need(f"{where}.mixer", data["mixer"], ("left", "right"))
        return cls(left=ZifunexAttention.from_json(f"{where}.mixer.left", mixer["left"]),
                   right=ZifunexScan.from_json(f"{where}.mixer.right", mixer["right"]), ff=ff)

    def to_json(self) -> dict[str, Any]:
        mixer = self.linear.to_json() if self.linear is not None else {"left": self.left.to_json(),
                                                                       "right": self.right.to_json()}
        return {"mixer": mixer, "mlp": None if self.ff is None else {"ff": self.ff, "kind": "dense"},
                "type": self.type}


@dataclass(frozen=True)
class ZifunexLoop:
    start: int
    stop: int
    times: int

    def __post_init__(self) -> None:
        for name in ("start", "stop", "times"):
            if type(getattr(self, name)) is not int:
                raise ConfigError(f"loop.{name} must be an integer")
        if not 0 <= self.start < self.stop or self.times < 1:
            raise ConfigError("a loop runs from start to stop - 1, at least one layer, at least once")


@dataclass(frozen=True)
class ZifunexBigram:
    buckets: int
    mul_prev: int
    mul_cur: int

    def __post_init__(self) -> None:
        _positive_int("embedding.bigram.buckets", self.buckets)
        for name in ("mul_prev", "mul_cur"):
            value = getattr(self, name)
            if type(value) is not int or value < 0 or value >= 1 << 31:
                raise ConfigError(f"embedding.bigram.{name} must be a non-negative 32-bit integer")


@dataclass(frozen=True)
class ZifunexConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int
    layers: tuple[ZifunexLayer, ...]
    bigram: ZifunexBigram | None = None
    loop: ZifunexLoop | None = None
    eos_token_ids: tuple[int, ...] = ()

    architecture = "Zifunex"

    def __post_init__(self) -> None:
        for name in ("vocab", "width", "streams"):
            _positive_int(name, getattr(self, name))
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        if self.loop is not None and self.loop.stop > len(self.layers):
            raise ConfigError("loop.stop must not exceed the number of layers")

    @classmethod
    def from_json(cls, data: Mapping[str, Any]) -> "ZifunexConfig":
        data = _need("config.json", data, ("vocab", "width", "norm", "streams", "layers"))
        norm = _need("config.json 'norm'", data["norm"], ("eps",))
        if not isinstance(data["layers"], list):
            raise ConfigError("config.json 'layers' must be a list")
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else (eos,) if type(eos) is int else tuple(eos)
        bigram = _need("embedding", data.get("embedding") or {}, ()).get("bigram")
        if bigram is not None:
            keys = ("buckets", "mul_prev", "mul_cur")
            bigram = ZifunexBigram(**{key: _need("embedding.bigram", bigram, keys)[key] for key in keys})
        loop = data.get("loop")
        if loop is not None:
            keys = ("start", "stop", "times")
            loop = ZifunexLoop(**{key: _need("loop", loop, keys)[key] for key in keys})
        return cls(vocab=data["vocab"], width=data["width"], norm_eps=_number("norm.eps", norm["eps"]),
                   streams=data["streams"],
                   layers=tuple(ZifunexLayer.from_json(i, layer) for i, layer in enumerate(data["layers"])),
                   bigram=bigram, loop=loop, eos_token_ids=eos_ids)

    def to_json(self) -> dict[str, Any]:
        data: dict[str, Any] = {"architecture": self.architecture,
                                "layers": [layer.to_json() for layer in self.layers],
                                "norm": {"eps": self.norm_eps}, "streams": self.streams, "vocab": self.vocab,
                                "width": self.width}
        if self.bigram is not None:
            data["embedding"] = {"bigram": {"buckets": self.bigram.buckets, "mul_cur": self.bigram.mul_cur,
                                            "mul_prev": self.bigram.mul_prev}}
        if self.loop is not None:
            data["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.eos_token_ids:
            data["eos_token_id"] = list(self.eos_token_ids)
        return data

    # ------------------------------------------------------------------ spec
    def run_order(self) -> tuple[int, ...]:
        """The layers in the order they run: a loop's stretch several times in a row."""
        every = tuple(range(len(self.layers)))
        if self.loop is None:
            return every
        start, stop = self.loop.start, self.loop.stop
        return every[:start] + every[start:stop] * self.loop.times + every[stop:]

    def _mixer_spec(self, layer: ZifunexLayer) -> PartSpec:
        if layer.linear is not None:
            linear = layer.linear
            return PartSpec("gated_linear_attention", {
                "hidden_size": self.width, "num_heads": linear.heads, "key_dim": linear.dim,
                "value_dim": linear.vdim, "query_scale": linear.dim ** -0.5, "decay_exponent": 1.0 / linear.tau,
                "out_norm": "weight", "eps": self.norm_eps, "gate": "silu", "float32_output": True})
        left, right = layer.left, layer.right
        position = None if not left.rot_dims else PartSpec(
            "rope_half_split_computed", {"dims": left.rot_dims, "base": left.rot_base})
        return PartSpec("parallel_mixers", {
            "hidden_size": self.width, "eps": self.norm_eps, "factor": 0.5,
            "left": PartSpec("windowed_attention", {
                "hidden_size": self.width, "num_heads": left.heads, "num_kv_heads": left.kv_heads,
                "key_dim": left.dim, "value_dim": left.vdim, "scale": left.scale, "softcap": left.softcap,
                "position": position, "qk_bias": True, "v_bias": True, "o_bias": True}),
            "right": PartSpec("selective_scan", {
                "hidden_size": self.width, "inner": right.inner, "state": right.state, "dt_rank": right.dt_rank,
                "taps": right.conv})})

    def to_spec(self) -> ModelSpec:
        norm = PartSpec("layer_norm_hyper32", {"width": self.width, "eps": self.norm_eps})
        block = PartSpec("hyper_residual", {
            "streams": self.streams, "mixer_norm_name": "norm1", "feed_forward_norm_name": "norm2",
            "mixer_connection_name": "hc1", "feed_forward_connection_name": "hc2", "mixer_name": "mix",
            "feed_forward_name": "mlp"})
        layers = []
        for index, layer in enumerate(self.layers):
            feed_forward = None
            if layer.ff is not None:
                feed_forward = PartSpec("gated_mlp", {
                    "hidden_size": self.width, "intermediate_size": layer.ff, "activation": "gelu_tanh",
                    "float32_output": True, "names": {"gate": "gate", "up": "up", "down": "down"}})
            layers.append(LayerSpec(prefix=f"l{index}", block=block, mixer=self._mixer_spec(layer),
                                    feed_forward=feed_forward, norm=norm))
        pairs = None if self.bigram is None else {
            "buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur,
            "name": "bigram"}
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width,
            max_positions=UNBOUNDED_POSITIONS,
            embedding=PartSpec("pair_embedding", {"vocab_size": self.vocab, "width": self.width, "name": "embed",
                                                  "pairs": pairs}),
            layers=tuple(layers), order=tuple(RunStep(index) for index in self.run_order()),
            final_norm=norm.with_params(name="final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "width": self.width, "tied_to": None,
                                      "name": "head"}),
            eos_token_ids=self.eos_token_ids)


register_architecture(ZifunexConfig.architecture, ZifunexConfig)
