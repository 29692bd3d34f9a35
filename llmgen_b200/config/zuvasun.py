"""Typed configuration of the Zuvasun decoder, read from its config.json.

    architecture      "Zuvasun"
    vocab, width      sizes of the table of embeddings and of the residual stream
    norm.eps          eps of every RMSNorm
    layers[i]         type: "attention" | "latent_attention"; mixer: that mixer's sizes and constants;
                      mlp: null or {kind: "moe", expert: {ff}, router: {experts, top, scale}}
    attention         heads, kv_heads, dim, vdim (equal to dim: the values are the projected keys), scale,
                      q_temp: {coef, every} (optional)
    latent_attention  heads, dim (unrotated), rot_dim (rotated), vdim, kv_rank, scale, mask: {size} (optional),
                      rot: {base, dims, scaling: {factor, original, fast, slow} (optional)},
                      kv_from: the layer whose cached entries this one reads (optional)

Every size and constant comes from the file; `max_positions` (rows of the rotary tables) is optional.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

from .base import ConfigReader
from .derupel import _sub

ATTENTION = "attention"
LATENT_ATTENTION = "latent_attention"
MOE = "moe"
DEFAULT_MAX_POSITIONS = 1 << 16


@dataclass(frozen=True)
class AttentionMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    q_temp: Optional[Tuple[float, float]]        # (coef, every)


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    scaling: Optional[Tuple[float, float, float, float]]   # (factor, original, fast, slow)


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int                                  # 0: every earlier key
    rot: RotationConfig
    kv_from: Optional[int]


@dataclass(frozen=True)
class MlpConfig:
    ff: int
    experts: int
    top: int
    scale: float


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: object
    mlp: Optional[MlpConfig]


def _attention(m: ConfigReader, r: ConfigReader, i: int) -> Optional[AttentionMixerConfig]:
    heads, kv_heads, dim = m.integer("heads"), m.integer("kv_heads"), m.integer("dim")
    vdim, scale = m.integer("vdim", default=dim), m.number("scale", positive=False)
    temp = _sub(m, "q_temp", m.where, required=False)
    coef = temp.number("coef", positive=False) if temp is not None else 0.0
    every = temp.number("every") if temp is not None else 1.0
    if None in (heads, kv_heads, dim, vdim, scale, coef, every):
        return None
    r.check(heads % kv_heads == 0, f"layers[{i}].mixer: {heads} heads are not a multiple of {kv_heads} kv_heads")
    r.check(vdim == dim, f"layers[{i}].mixer: the values are the keys, so vdim {vdim} must equal dim {dim}")
    return AttentionMixerConfig(heads, kv_heads, dim, scale, (coef, every) if temp is not None else None)


def _latent(m: ConfigReader, r: ConfigReader, i: int) -> Optional[LatentMixerConfig]:
    heads, dim, rot_dim, vdim = m.integer("heads"), m.integer("dim"), m.integer("rot_dim"), m.integer("vdim")
    kv_rank, scale = m.integer("kv_rank"), m.number("scale", positive=False)
    mask = _sub(m, "mask", m.where, required=False)
    window = mask.integer("size") if mask is not None else 0
    rot = _sub(m, "rot", m.where)
    if rot is None:
        return None
    base, dims = rot.number("base"), rot.integer("dims", default=rot_dim)
    sc = _sub(rot, "scaling", rot.where, required=False)
    scaling = None
    if sc is not None:
        scaling = tuple(sc.number(k) for k in ("factor", "original", "fast", "slow"))
    kv_from = m.integer("kv_from", default=-1, minimum=-1)
    if None in (heads, dim, rot_dim, vdim, kv_rank, scale, window, base, dims, kv_from) or (scaling is not None and None in scaling):
        return None
    r.check(rot_dim % 2 == 0 and dims == rot_dim, f"layers[{i}].mixer: rot.dims {dims} must equal rot_dim {rot_dim}, an even number")
    r.check(scaling is None or base > 1.0, f"layers[{i}].mixer.rot: scaled frequencies need a base above 1, got {base}")
    return LatentMixerConfig(heads, dim, rot_dim, vdim, kv_rank, scale, window, RotationConfig(base, dims, scaling),
                             kv_from if kv_from >= 0 else None)


def _layer(data, i: int, r: ConfigReader, where: str) -> Optional[LayerConfig]:
    if not isinstance(data, dict):
        r.problem(f"layers[{i}] must be an object")
        return None
    n0 = len(r.problems)
    lr = ConfigReader(data, f"{where}.layers[{i}]")
    lr.problems = r.problems
    kind = lr.string("type", choices=(ATTENTION, LATENT_ATTENTION))
    m = _sub(lr, "mixer", lr.where)
    mixer = None
    if m is not None and kind == ATTENTION:
        mixer = _attention(m, r, i)
    elif m is not None and kind == LATENT_ATTENTION:
        mixer = _latent(m, r, i)
    mlp = None
    if data.get("mlp") is not None:
        f = _sub(lr, "mlp", lr.where)
        if f is not None and f.string("kind", choices=(MOE,)) is not None:
            e, ro = _sub(f, "expert", f.where), _sub(f, "router", f.where)
            ff = e.integer("ff") if e is not None else None
            experts = ro.integer("experts") if ro is not None else None
            top = ro.integer("top") if ro is not None else None
            scale = ro.number("scale", default=1.0, positive=False) if ro is not None else None
            if None not in (ff, experts, top, scale):
                r.check(top <= experts, f"layers[{i}].mlp.router: top {top} of {experts} experts")
                mlp = MlpConfig(ff, experts, top, scale)
    if len(r.problems) > n0 or kind is None or mixer is None:
        return None
    return LayerConfig(kind, mixer, mlp)


def _check_readers(layers: List[Optional[LayerConfig]], r: ConfigReader) -> None:
    """A layer that reads another's entries: that layer comes before it, keeps entries of its own, and they fit."""
    for i, layer in enumerate(layers):
        src = getattr(layer.mixer, "kv_from", None) if layer is not None else None
        if src is None:
            continue
        owner = layers[src] if src < i else None
        if owner is None:
            r.problem(f"layers[{i}].mixer.kv_from {src} must name an earlier layer")
        elif owner.type != LATENT_ATTENTION or owner.mixer.kv_from is not None:
            r.problem(f"layers[{i}].mixer.kv_from {src}: that layer keeps no latent entries of its own")
        elif (owner.mixer.kv_rank, owner.mixer.rot_dim, owner.mixer.rot) != (layer.mixer.kv_rank, layer.mixer.rot_dim, layer.mixer.rot):
            r.problem(f"layers[{i}].mixer.kv_from {src}: kv_rank, rot_dim and rot of the two layers differ")


@dataclass(frozen=True)
class ZuvasunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[LayerConfig, ...]
    max_positions: int
    raw: dict

    architecture = "Zuvasun"

    @classmethod
    def from_dict(cls, data: dict, where: str = "config.json") -> "ZuvasunConfig":
        r = ConfigReader(data, where)
        vocab, width = r.integer("vocab"), r.integer("width")
        norm = _sub(r, "norm", where)
        eps = norm.number("eps") if norm is not None else None
        max_positions = r.integer("max_positions", default=DEFAULT_MAX_POSITIONS)
        layers = r.raw("layers")
        parsed: List[Optional[LayerConfig]] = []
        if not isinstance(layers, list) or not layers:
            r.problem("'layers' must be a non-empty list")
        else:
            parsed = [_layer(d, i, r, where) for i, d in enumerate(layers)]
            _check_readers(parsed, r)
        r.finish()
        return cls(vocab, width, eps, tuple(parsed), max_positions, dict(data))

    def to_dict(self) -> dict:
        return dict(self.raw)
