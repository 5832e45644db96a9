"""Typed configuration of the Boketar decoder: pre-norm layers on a residual of several streams (hyper-connections),
whose mixers are a delta rule with a decay per key channel (``channel_delta``) or softmax attention behind a sliding
window with a sink beside lightning attention (``parallel``), with dense feed-forwards (or none).

config.json gives every size and constant: ``vocab``, ``width``, ``streams``, ``norm`` ``{eps}``, ``embedding``
``{scale}`` and ``layers``, a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``.  Two sizes are not in config.json but
in the tensors' shapes: the inner widths of the narrow pairs of products that form the decays (``decay_rank``) and the
output gate (``gate_rank``) of a delta layer (config.json may name them, and a folder of random weights written from a
configuration does).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Mapping, Optional, Tuple

from .gezozen_config import DeltaMixerConfig, RotationConfig, SoftmaxSideConfig
from .model_config import ConfigError
from .viresun_config import _float, _int

ShapeOf = Optional[Callable[[str], Optional[Tuple[int, ...]]]]


@dataclass(frozen=True)
class WindowSideConfig(SoftmaxSideConfig):
    """The attention side of a pair: the sizes any softmax side has, and the taps of its short convolutions."""
    conv: int = 1

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "WindowSideConfig":
        base = SoftmaxSideConfig.from_dict(d, where)
        if base.softcap is not None or base.rot.scaling is not None:
            raise ConfigError(f"{where}: neither a soft cap nor a stretched rotation belongs to this design")
        if base.window is not None and base.window < 1:
            raise ConfigError(f"{where}.mask.size must be positive")
        return cls(**vars(base), conv=_int(d, "conv", where, minimum=1))


@dataclass(frozen=True)
class LightningSideConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "LightningSideConfig":
        heads, dim, decay = _int(d, "heads", where), _int(d, "dim", where), d.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or not all(isinstance(v, (int, float)) for v in decay):
            raise ConfigError(f"{where}.decay must list one number per head")
        return cls(heads=heads, dim=dim, vdim=_int(d, "vdim", where) if d.get("vdim") is not None else dim,
                   decay=tuple(float(v) for v in decay))


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: WindowSideConfig
    right: LightningSideConfig


@dataclass(frozen=True)
class ChannelDeltaMixerConfig(DeltaMixerConfig):
    decay_rank: int = 0
    gate_rank: int = 0

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str, layer: int, shape_of: ShapeOf) -> "ChannelDeltaMixerConfig":
        base = DeltaMixerConfig.from_dict(d, where)
        if base.conv < 1:
            raise ConfigError(f"{where}.conv must be at least 1")

        def rank(key: str, tensor: str) -> int:
            if d.get(key) is not None:
                return _int(d, key, where, minimum=1)
            shape = shape_of(f"l{layer}.mix.{tensor}") if shape_of is not None else None
            if not shape:
                raise ConfigError(f"{where}.{key} is neither in the configuration nor to be read off a tensor's shape")
            return int(shape[0])
        return cls(**vars(base), decay_rank=rank("decay_rank", "a1"), gate_rank=rank("gate_rank", "g1"))


@dataclass(frozen=True)
class BoketarLayerConfig:
    type: str                    # "channel_delta" | "parallel"
    mixer: Any                   # ChannelDeltaMixerConfig | ParallelMixerConfig
    ff: Optional[int]            # inner width of the dense feed-forward, None: the layer has none


@dataclass(frozen=True)
class BoketarConfig:
    vocab_size: int
    hidden_size: int
    streams: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[BoketarLayerConfig, ...]
    tie_word_embeddings: bool = False
    torch_dtype: str = "bfloat16"
    max_position_embeddings: int = 1 << 17      # the design sets no limit; block tables are made this wide

    #: ``from_dict`` takes ``shape_of`` (tensor name -> shape or None) for the sizes the tensors hold
    wants_tensor_shapes = True

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], shape_of: ShapeOf = None) -> "BoketarConfig":
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a list with at least one entry")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind, m = L.get("type"), L.get("mixer") or {}
            if kind == "channel_delta":
                mixer = ChannelDeltaMixerConfig.from_dict(m, where + ".mixer", i, shape_of)
            elif kind == "parallel":
                mixer = ParallelMixerConfig(WindowSideConfig.from_dict(m.get("left") or {}, where + ".mixer.left"),
                                            LightningSideConfig.from_dict(m.get("right") or {}, where + ".mixer.right"))
            else:
                raise ConfigError(f"{where}.type {kind!r} is not known (channel_delta, parallel)")
            mlp, ff = L.get("mlp"), None
            if mlp:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}.mlp.kind {mlp.get('kind')!r} is not known (dense)")
                ff = _int(mlp, "ff", where + ".mlp", minimum=1)
            layers.append(BoketarLayerConfig(kind, mixer, ff))
        eps = _float(d.get("norm") or {}, "eps", "norm")
        if not eps > 0:
            raise ConfigError("norm.eps must be positive")
        emb = d.get("embedding") or {}
        dtype = str(d.get("torch_dtype", d.get("dtype", "bfloat16")) or "bfloat16").replace("torch.", "")
        return cls(vocab_size=_int(d, "vocab", "config"), hidden_size=_int(d, "width", "config"),
                   streams=_int(d, "streams", "config", minimum=1), norm_eps=eps,
                   embedding_scale=_float(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0,
                   layers=tuple(layers), torch_dtype=dtype,
                   max_position_embeddings=_int(d, "max_position_embeddings", "config")
                   if d.get("max_position_embeddings") is not None else 1 << 17)
