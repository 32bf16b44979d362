"""Typed configuration of the Sefelorn decoder, read from its own config.json keys.

    architecture: "Sefelorn"; vocab; width; norm: {eps}; embedding: {scale} (absent: 1); logit_scale (absent: 1);
    layers: [{type: "mamba2" | "parallel", mixer: {...}, mlp: null | {kind: "dense", ff, limit}}, ...];
    loop: null | {start (absent: 0), stop, times} (absent: every layer runs once); max_positions (optional).
    mamba2 mixer:   heads, vdim, state, groups (absent: 1), conv (taps), norm_groups (absent: 1)
    parallel mixer: left_scale, right_scale (absent: 1);
        left:  heads, kv_heads (absent: heads), dim, vdim (absent: dim), scale (absent: dim^-1/2), rot: null | {base, dims},
               mask: null | {size (absent: every key), keep_first (absent: 0)}
        right: heads, dim, vdim (absent: dim), tau

One size is not in config.json but in the checkpoint's tensor shapes: the inner width of the right mixer's low-rank map
(rows of ``l<i>.mix.right.a1``); :meth:`SefelornConfig.resolve_shapes` takes it from there.  A configuration for random
weights may name it itself (``decay_rank`` in ``right``).  Every size and constant lives here and reaches the parts as
parameters.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError, _require

MAMBA2 = "mamba2"
PARALLEL = "parallel"
DEFAULT_MAX_POSITIONS = 1 << 20


@dataclass(frozen=True)
class Mamba2MixerConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                          # taps of the short convolution
    norm_groups: int


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int                      # 0: no rotation
    rot_base: float
    window: Optional[int]              # None: every key
    keep_first: int                    # a sequence's first keys that stay visible


@dataclass(frozen=True)
class LinearAttentionConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int]          # None: not known yet (the checkpoint says)


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: WindowAttentionConfig
    right: LinearAttentionConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SefelornLayerConfig:
    type: str
    mixer: Any
    ff: Optional[int]                  # inner width of the dense feed-forward; None: the layer has none
    limit: float                       # of the clamped gate


def _opt(d: Mapping[str, Any], key: str, typ, where: str, default):
    return _require(d, key, typ, where) if d.get(key) is not None else default


def _object(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where}: missing required object '{key}'")
    return v


def _mamba2(m: Mapping[str, Any], w: str) -> Mamba2MixerConfig:
    c = Mamba2MixerConfig(_require(m, "heads", int, w), _require(m, "vdim", int, w), _require(m, "state", int, w),
                          _opt(m, "groups", int, w, 1), _require(m, "conv", int, w), _opt(m, "norm_groups", int, w, 1))
    if c.heads % c.groups:
        raise ConfigError(f"{w}: {c.heads} heads are not a multiple of {c.groups} groups")
    if c.heads * c.vdim % c.norm_groups:
        raise ConfigError(f"{w}: {c.heads} heads of {c.vdim} do not divide into {c.norm_groups} norm_groups")
    return c


def _left(m: Mapping[str, Any], w: str) -> WindowAttentionConfig:
    heads, dim = _require(m, "heads", int, w), _require(m, "dim", int, w)
    rot, mask = m.get("rot"), m.get("mask")
    dims, base = 0, 1.0
    if isinstance(rot, Mapping):
        dims, base = _require(rot, "dims", int, w + " rot"), _require(rot, "base", float, w + " rot")
    window, keep = None, 0
    if isinstance(mask, Mapping):
        window = _opt(mask, "size", int, w + " mask", None)
        keep = mask.get("keep_first") or 0
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ConfigError(f"{w} mask: 'keep_first' must be an integer that is not negative, got {keep!r}")
    c = WindowAttentionConfig(heads, _opt(m, "kv_heads", int, w, heads), dim, _opt(m, "vdim", int, w, dim),
                              _opt(m, "scale", float, w, float(dim) ** -0.5), dims, base, window, keep)
    if c.heads % c.kv_heads:
        raise ConfigError(f"{w}: {c.heads} heads are not a multiple of {c.kv_heads} kv_heads")
    if dims % 2 or dims > dim:
        raise ConfigError(f"{w}: rot.dims {dims} must be even and at most dim {dim}")
    return c


def _right(m: Mapping[str, Any], w: str) -> LinearAttentionConfig:
    dim = _require(m, "dim", int, w)
    c = LinearAttentionConfig(_require(m, "heads", int, w), dim, _opt(m, "vdim", int, w, dim), _require(m, "tau", float, w),
                              _opt(m, "decay_rank", int, w, None))
    if not c.tau > 0:
        raise ConfigError(f"{w}: 'tau' must be positive, got {c.tau}")
    return c


@dataclass(frozen=True)
class SefelornConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[SefelornLayerConfig, ...]
    loop: Optional[Tuple[int, int, int]]        # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS
    raw: Optional[Mapping[str, Any]] = None     # the mapping it was read from, for writing it back

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str = "config.json") -> "SefelornConfig":
        vocab, width = _require(d, "vocab", int, where), _require(d, "width", int, where)
        eps = _require(_object(d, "norm", where), "eps", float, where + " norm")
        emb = d.get("embedding")
        emb_scale = _opt(emb, "scale", float, where + " embedding", 1.0) if isinstance(emb, Mapping) else 1.0
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must list at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            w = f"{where} layers[{i}]"
            if not isinstance(L, Mapping):
                raise ConfigError(f"{w}: a layer is an object with 'type', 'mixer' and 'mlp'")
            m, kind = _object(L, "mixer", w), L.get("type")
            if kind == MAMBA2:
                mixer = _mamba2(m, w)
            elif kind == PARALLEL:
                mixer = ParallelMixerConfig(_left(_object(m, "left", w), w + " left"), _right(_object(m, "right", w), w + " right"),
                                            _opt(m, "left_scale", float, w, 1.0), _opt(m, "right_scale", float, w, 1.0))
            else:
                raise ConfigError(f"{w}: unknown layer type {kind!r} (known: {MAMBA2}, {PARALLEL})")
            mlp = L.get("mlp")
            ff, limit = None, 0.0
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise ConfigError(f"{w}: 'mlp' must be an object or null")
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{w}: unknown mlp kind {mlp.get('kind')!r} (known: dense)")
                ff, limit = _require(mlp, "ff", int, w + " mlp"), _require(mlp, "limit", float, w + " mlp")
                if not limit > 0:
                    raise ConfigError(f"{w} mlp: 'limit' must be positive, got {limit}")
            layers.append(SefelornLayerConfig(kind, mixer, ff, limit))
        loop = d.get("loop")
        loop_t = None
        if isinstance(loop, Mapping):
            start = loop.get("start", 0)
            stop, times = _require(loop, "stop", int, where + " loop"), _require(loop, "times", int, where + " loop")
            if isinstance(start, bool) or not isinstance(start, int) or not 0 <= start < stop <= len(layers):
                raise ConfigError(f"{where}: loop start {start!r} .. stop {stop} does not lie within the {len(layers)} layers")
            loop_t = (start, stop, times)
        max_pos = d.get("max_positions", DEFAULT_MAX_POSITIONS)
        if isinstance(max_pos, bool) or not isinstance(max_pos, int) or max_pos <= 0:
            raise ConfigError(f"{where}: 'max_positions' must be a positive integer, got {max_pos!r}")
        return cls(vocab=vocab, width=width, eps=float(eps), embedding_scale=float(emb_scale),
                   logit_scale=float(_opt(d, "logit_scale", float, where, 1.0)), layers=tuple(layers), loop=loop_t,
                   max_positions=max_pos, raw=dict(d))

    def resolve_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "SefelornConfig":
        """The sizes that only the checkpoint's tensor shapes give (name → shape)."""
        layers = []
        for i, L in enumerate(self.layers):
            name = f"l{i}.mix.right.a1"
            if L.type == PARALLEL and L.mixer.right.decay_rank is None and len(shapes.get(name, ())) == 2:
                L = replace(L, mixer=replace(L.mixer, right=replace(L.mixer.right, decay_rank=int(shapes[name][0]))))
            layers.append(L)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        if self.raw is not None:
            return dict(self.raw)
        raise ValueError("this configuration was not read from a mapping")
