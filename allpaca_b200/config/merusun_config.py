"""Typed configuration of the Merusun decoder: layers with a norm before and after every sublayer, whose mixers are a
matrix memory (``mlstm``), attention through a shared latent with a rotated key part behind a sliding window
(``latent_attention``) or grouped-query attention without positions behind a sliding window, with one added to the
softmax's denominator (``attention``, which may read the keys and values an earlier layer keeps), with routed experts
(chosen among the best groups of neighbouring experts) and a shared expert, or no feed-forward.

config.json gives every size and constant: ``vocab``, ``width``, ``norm`` ``{eps}``, ``embedding`` ``{scale}`` and
``layers``, a list of ``{"type", "mixer": {...}, "mlp": {...} | null}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .gezozen_config import RotationConfig
from .model_config import ConfigError
from .viresun_config import _float, _int


def _window(d: Mapping[str, Any], where: str) -> Optional[int]:
    mask = d.get("mask") or None
    if not mask or mask.get("size") is None:
        return None
    return _int(mask, "size", where + ".mask", minimum=1)


def _value_size(d: Mapping[str, Any], where: str, dim: int) -> int:
    return _int(d, "vdim", where) if d.get("vdim") is not None else dim


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "MatrixMemoryConfig":
        dim, cap = _int(d, "dim", where), _float(d, "gate_cap", where)
        if not cap > 0:
            raise ConfigError(f"{where}.gate_cap must be positive")
        return cls(heads=_int(d, "heads", where), dim=dim, vdim=_value_size(d, where, dim), gate_cap=cap)


@dataclass(frozen=True)
class WindowedLatentConfig:
    heads: int
    dim: int                    # unrotated query/key dimensions per head
    rot_dim: int                # rotated ones; the key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot: RotationConfig
    window: Optional[int]       # mask.size

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "WindowedLatentConfig":
        dim, rot_dim = _int(d, "dim", where), _int(d, "rot_dim", where)
        if d.get("kv_from") is not None:
            raise ConfigError(f"{where}.kv_from: a latent attention layer of this design keeps a latent of its own")
        rot = RotationConfig.from_dict(d.get("rot") or {}, where + ".rot", rot_dim)
        if rot.scaling is not None:
            raise ConfigError(f"{where}.rot.scaling: a stretched rotation does not belong to this design")
        return cls(heads=_int(d, "heads", where), dim=dim, rot_dim=rot_dim, vdim=_value_size(d, where, dim),
                   kv_rank=_int(d, "kv_rank", where), scale=_float(d, "scale", where), rot=rot,
                   window=_window(d, where))


@dataclass(frozen=True)
class WindowedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]       # mask.size
    kv_from: Optional[int]      # the layer whose keys and values this one reads

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "WindowedAttentionConfig":
        heads = _int(d, "heads", where)
        kv = _int(d, "kv_heads", where) if d.get("kv_heads") is not None else heads
        if heads % kv:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv} kv_heads")
        dim = _int(d, "dim", where)
        return cls(heads=heads, kv_heads=kv, dim=dim, vdim=_value_size(d, where, dim), scale=_float(d, "scale", where),
                   window=_window(d, where),
                   kv_from=_int(d, "kv_from", where, minimum=0) if d.get("kv_from") is not None else None)


@dataclass(frozen=True)
class GroupRoutedConfig:
    ff: int
    experts: int
    top: int
    scale: float
    groups: int                 # equal groups of neighbouring experts ...
    keep: int                   # ... of which a row chooses within this many
    shared_ff: Optional[int]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "GroupRoutedConfig":
        if d.get("kind") != "moe":
            raise ConfigError(f"{where}.kind {d.get('kind')!r} is not known (moe)")
        expert, r, shared = d.get("expert") or {}, d.get("router") or {}, d.get("shared") or None
        w = where + ".router"
        groups = r.get("groups") or None
        out = cls(ff=_int(expert, "ff", where + ".expert"), experts=_int(r, "experts", w), top=_int(r, "top", w),
                  scale=_float(r, "scale", w) if r.get("scale") is not None else 1.0,
                  groups=_int(groups, "count", w + ".groups") if groups else 1,
                  keep=_int(groups, "keep", w + ".groups") if groups else 1,
                  shared_ff=_int(shared, "ff", where + ".shared") if shared else None)
        if out.experts % out.groups or out.keep > out.groups:
            raise ConfigError(f"{w}: {out.experts} experts do not fall into {out.groups} equal groups, of which "
                              f"{out.keep} are kept")
        if out.top > out.experts // out.groups * out.keep:
            raise ConfigError(f"{w}: {out.top} experts cannot be chosen among those of {out.keep} of {out.groups} groups")
        return out


@dataclass(frozen=True)
class MerusunLayerConfig:
    type: str                   # "mlstm" | "latent_attention" | "attention"
    mixer: Any                  # MatrixMemoryConfig | WindowedLatentConfig | WindowedAttentionConfig
    mlp: Optional[GroupRoutedConfig]


_MIXERS = {"mlstm": MatrixMemoryConfig, "latent_attention": WindowedLatentConfig, "attention": WindowedAttentionConfig}


@dataclass(frozen=True)
class MerusunConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[MerusunLayerConfig, ...]
    tie_word_embeddings: bool = False
    torch_dtype: str = "bfloat16"
    max_position_embeddings: int = 1 << 17      # the design sets no limit; block tables are made this wide

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MerusunConfig":
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers must be a list with at least one entry")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = L.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type {kind!r} is not known ({', '.join(_MIXERS)})")
            mixer = _MIXERS[kind].from_dict(L.get("mixer") or {}, where + ".mixer")
            j = getattr(mixer, "kv_from", None)
            if j is not None:
                if j >= i or layers[j].type != "attention" or layers[j].mixer.kv_from is not None:
                    raise ConfigError(f"{where}.mixer.kv_from must name an earlier attention layer that has key and "
                                      f"value projections of its own")
                src = layers[j].mixer
                if (src.heads, src.kv_heads, src.dim, src.vdim) != (mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ConfigError(f"{where} reads what layer {j} keeps, but their head counts or sizes differ")
            layers.append(MerusunLayerConfig(kind, mixer, GroupRoutedConfig.from_dict(L["mlp"], where + ".mlp")
                                             if L.get("mlp") else None))
        eps = _float(d.get("norm") or {}, "eps", "norm")
        if not eps > 0:
            raise ConfigError("norm.eps must be positive")
        emb = d.get("embedding") or {}
        dtype = str(d.get("torch_dtype", d.get("dtype", "bfloat16")) or "bfloat16").replace("torch.", "")
        return cls(vocab_size=_int(d, "vocab", "config"), hidden_size=_int(d, "width", "config"), norm_eps=eps,
                   embedding_scale=_float(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0,
                   layers=tuple(layers), torch_dtype=dtype,
                   max_position_embeddings=_int(d, "max_position_embeddings", "config")
                   if d.get("max_position_embeddings") is not None else 1 << 17)

    def cache_window(self, i: int) -> Optional[int]:
        """How far back the keys and values layer ``i`` keeps must stay readable: the largest window among the layer
        and the layers that read them (None as soon as one of them has no window)."""
        windows = [self.layers[i].mixer.window] + [L.mixer.window for L in self.layers
                                                   if getattr(L.mixer, "kv_from", None) == i]
        return None if any(w is None for w in windows) else max(windows)
