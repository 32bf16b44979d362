"""Typed configuration of the Gemodra decoder, read from its own config.json keys.

    architecture: "Gemodra"; vocab; width; norm: {eps}; residual_mult (absent: 1); token_side: {dim} (absent: no per-layer
    token input); logit_softcap (absent: none); max_positions (optional);
    layers: [{type: "latent_attention" | "latent_attention_2", mixer: {...}, mlp: null | {...}}, ...]
    mixer:  heads, dim, vdim (absent: dim), kv_rank, q_rank, scale (absent: (dim + rot_dim)^-1/2), and for
            "latent_attention" rot_dim and rot: {base, dims}
    mlp:    kind "moe", expert: {ff}, router: {experts, top, identity (absent: 0), scale (absent: 1),
            groups: null | {count, keep}}, shared: null | {ff}

Every size and constant lives here and reaches the parts as parameters.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .model_config import ConfigError, _require

LATENT_ATTENTION = "latent_attention"
LATENT_ATTENTION_2 = "latent_attention_2"
DEFAULT_MAX_POSITIONS = 1 << 20


@dataclass(frozen=True)
class GemodraMixerConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_dim: int                       # 0: no rotated part
    rot_dims: int                      # coordinates of the rotated part that turn
    rot_base: float


@dataclass(frozen=True)
class GemodraMoeConfig:
    experts: int
    identity: int
    top: int
    expert_ff: int
    route_scale: float
    groups: Optional[Tuple[int, int]]  # (count, keep)
    shared_ff: Optional[int]


@dataclass(frozen=True)
class GemodraLayerConfig:
    type: str
    mixer: GemodraMixerConfig
    mlp: Optional[GemodraMoeConfig]


def _object(d: Mapping[str, Any], key: str, w: str, required: bool = False) -> Optional[Mapping[str, Any]]:
    v = d.get(key)
    if v is None and not required:
        return None
    if not isinstance(v, Mapping):
        raise ConfigError(f"{w}: '{key}' must be an object" + ("" if required else " or null"))
    return v


def _number(d: Mapping[str, Any], key: str, kind: type, default, w: str):
    return _require(d, key, kind, w) if d.get(key) is not None else default


def _count(d: Mapping[str, Any], key: str, w: str) -> int:
    """A whole number that may be 0; absent or null: 0."""
    v = d.get(key)
    if v is None:
        return 0
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"{w}: '{key}' must be a whole number from 0 on, got {v!r}")
    return v


def _mixer(kind: Any, m: Mapping[str, Any], w: str) -> GemodraMixerConfig:
    if kind not in (LATENT_ATTENTION, LATENT_ATTENTION_2):
        raise ConfigError(f"{w}: unknown layer type {kind!r} (known: {LATENT_ATTENTION}, {LATENT_ATTENTION_2})")
    heads, dim = _require(m, "heads", int, w), _require(m, "dim", int, w)
    rot_dim, rot_dims, rot_base = 0, 0, 0.0
    if kind == LATENT_ATTENTION:
        rot_dim = _require(m, "rot_dim", int, w)
        rot = _object(m, "rot", w, required=True)
        rot_dims, rot_base = _number(rot, "dims", int, rot_dim, w + " rot"), _require(rot, "base", float, w + " rot")
        if rot_dims % 2 or rot_dims > rot_dim:
            raise ConfigError(f"{w}: rot.dims {rot_dims} must be even and at most rot_dim {rot_dim}")
        if rot_base <= 0:
            raise ConfigError(f"{w}: rot.base must be positive")
    return GemodraMixerConfig(heads, dim, _number(m, "vdim", int, dim, w), _require(m, "kv_rank", int, w),
                              _require(m, "q_rank", int, w), _number(m, "scale", float, float(dim + rot_dim) ** -0.5, w),
                              rot_dim, rot_dims, rot_base)


def _mlp(mlp: Any, w: str) -> Optional[GemodraMoeConfig]:
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping):
        raise ConfigError(f"{w}: 'mlp' must be an object or null")
    if mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"{w}: unknown mlp kind {mlp.get('kind')!r} (known: moe)")
    router, expert = _object(mlp, "router", w, required=True), _object(mlp, "expert", w, required=True)
    experts, top = _require(router, "experts", int, w + " router"), _require(router, "top", int, w + " router")
    identity = _count(router, "identity", w + " router")
    n = experts + identity
    if top > n:
        raise ConfigError(f"{w}: top {top} of {n} experts")
    groups = _object(router, "groups", w + " router")
    if groups is not None:
        groups = (_require(groups, "count", int, w + " groups"), _require(groups, "keep", int, w + " groups"))
        if n % groups[0] or groups[1] > groups[0] or top > groups[1] * (n // groups[0]):
            raise ConfigError(f"{w}: {groups[0]} groups of {n} experts with {groups[1]} kept cannot give {top} experts")
    shared = _object(mlp, "shared", w)
    return GemodraMoeConfig(experts, identity, top, _require(expert, "ff", int, w + " expert"),
                            float(_number(router, "scale", float, 1.0, w + " router")), groups,
                            _require(shared, "ff", int, w + " shared") if shared is not None else None)


@dataclass(frozen=True)
class GemodraConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    side_dim: Optional[int]                     # columns of the token table per layer; None: no per-layer token input
    logit_softcap: Optional[float]
    layers: Tuple[GemodraLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    raw: Optional[Mapping[str, Any]] = None     # the mapping it was read from, for writing it back

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str = "config.json") -> "GemodraConfig":
        vocab = _require(d, "vocab", int, where)
        width = _require(d, "width", int, where)
        eps = _require(_object(d, "norm", where, required=True), "eps", float, where + " norm")
        side = _object(d, "token_side", where)
        cap = _number(d, "logit_softcap", float, None, where)
        if cap is not None and cap <= 0:
            raise ConfigError(f"{where}: 'logit_softcap' must be positive, got {cap}")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must list at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            w = f"{where} layers[{i}]"
            if not isinstance(L, Mapping) or not isinstance(L.get("mixer"), Mapping):
                raise ConfigError(f"{w}: a layer is an object with 'type', 'mixer' and 'mlp'")
            layers.append(GemodraLayerConfig(L.get("type"), _mixer(L.get("type"), L["mixer"], w), _mlp(L.get("mlp"), w)))
        max_pos = d.get("max_positions", DEFAULT_MAX_POSITIONS)
        if isinstance(max_pos, bool) or not isinstance(max_pos, int) or max_pos <= 0:
            raise ConfigError(f"{where}: 'max_positions' must be a positive integer, got {max_pos!r}")
        return cls(vocab=vocab, width=width, eps=float(eps), residual_mult=float(_number(d, "residual_mult", float, 1.0, where)),
                   side_dim=_require(side, "dim", int, where + " token_side") if side is not None else None,
                   logit_softcap=None if cap is None else float(cap), layers=tuple(layers), max_positions=max_pos, raw=dict(d))

    def to_dict(self) -> dict:
        if self.raw is not None:
            return dict(self.raw)
        raise ValueError("this configuration was not read from a mapping")
