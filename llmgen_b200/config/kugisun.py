"""Typed configuration of the Kugisun decoder, read from its config.json.

    architecture      "Kugisun"
    vocab, width      sizes of the table of embeddings (which is also the output matrix) and of the residual stream
    max_positions     rows of the table of learned positions: the longest sequence the model takes (optional in a model folder,
                      where the table's shape gives it)
    norm.eps          eps of every RMSNorm
    streams           number of residual streams per token (optional; absent: one plain stream)
    layers[i]         type: "parallel"; mixer: its sizes and constants; mlp: null, {kind: "dense", ff} or {kind: "moe",
                      expert: {ff}, router: {...}, shared: {ff} (optional)}; weights_of: j (optional): the layer has no tensors
                      of its own and uses layer j's, with a cache and a state of its own
    mixer             left: {heads, kv_heads, dim, vdim, scale, rot: {base, dims} (optional)}, right: {heads, kv_heads, dim, vdim,
                      conv (taps)}, left_scale, right_scale
    router            experts, top, scale (optional, 1), identity (optional, 0: outputs of the router behind the experts whose
                      result is the input itself), groups: {count, keep} (optional)

Every size and constant comes from the file.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigReader
from .derupel import _sub

PARALLEL = "parallel"
DENSE = "dense"
MOE = "moe"


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int           # 0: no rotation


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int               # taps


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: AttentionConfig
    right: DeltaConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MlpConfig:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    identity: int = 0
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0      # 0: no shared expert


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: ParallelMixerConfig
    mlp: Optional[MlpConfig]
    weights_of: Optional[int] = None


def _left(m: ConfigReader, r: ConfigReader, i: int) -> Optional[AttentionConfig]:
    a = _sub(m, "left", m.where)
    if a is None:
        return None
    heads, kv_heads, dim, vdim, scale = a.integer("heads"), a.integer("kv_heads"), a.integer("dim"), a.integer("vdim"), a.number("scale", positive=False)
    rot = _sub(a, "rot", a.where, required=False)
    base = rot.number("base") if rot is not None else 1.0
    dims = rot.integer("dims", minimum=0) if rot is not None else 0
    if None in (heads, kv_heads, dim, vdim, scale, base, dims):
        return None
    r.check(heads % kv_heads == 0, f"layers[{i}].mixer.left: {heads} heads are not a multiple of {kv_heads} kv_heads")
    r.check(dims % 2 == 0 and dims <= dim, f"layers[{i}].mixer.left.rot.dims {dims} must be even and at most dim {dim}")
    return AttentionConfig(heads, kv_heads, dim, vdim, scale, base, dims)


def _right(m: ConfigReader, r: ConfigReader, i: int) -> Optional[DeltaConfig]:
    d = _sub(m, "right", m.where)
    if d is None:
        return None
    heads, kv_heads, dim, vdim, conv = d.integer("heads"), d.integer("kv_heads"), d.integer("dim"), d.integer("vdim"), d.integer("conv")
    if None in (heads, kv_heads, dim, vdim, conv):
        return None
    r.check(heads % kv_heads == 0, f"layers[{i}].mixer.right: {heads} heads are not a multiple of {kv_heads} kv_heads")
    r.check(conv <= 8, f"layers[{i}].mixer.right.conv {conv} taps: at most 8")
    return DeltaConfig(heads, kv_heads, dim, vdim, conv)


def _mlp(lr: ConfigReader, r: ConfigReader, i: int) -> Optional[MlpConfig]:
    f = _sub(lr, "mlp", lr.where)
    if f is None:
        return None
    kind = f.string("kind", choices=(DENSE, MOE))
    if kind == DENSE:
        ff = f.integer("ff")
        return MlpConfig(kind, ff) if ff is not None else None
    if kind != MOE:
        return None
    e, ro, sh = _sub(f, "expert", f.where), _sub(f, "router", f.where), _sub(f, "shared", f.where, required=False)
    if e is None or ro is None:
        return None
    groups = _sub(ro, "groups", ro.where, required=False)
    count = groups.integer("count") if groups is not None else 1
    keep = groups.integer("keep") if groups is not None else 1
    ff, experts, top = e.integer("ff"), ro.integer("experts"), ro.integer("top")
    scale, identity = ro.number("scale", default=1.0, positive=False), ro.integer("identity", default=0, minimum=0)
    shared_ff = sh.integer("ff") if sh is not None else 0
    if None in (ff, experts, top, scale, identity, count, keep, shared_ff):
        return None
    outputs = experts + identity
    r.check(outputs % count == 0, f"layers[{i}].mlp.router: {outputs} outputs do not form {count} equal groups")
    r.check(keep <= count, f"layers[{i}].mlp.router.groups: {keep} of {count} groups")
    r.check(top <= outputs // count * keep, f"layers[{i}].mlp.router: top {top} of {outputs // count * keep} outputs in the groups kept")
    return MlpConfig(kind, ff, experts, top, scale, identity, count, keep, shared_ff)


def _layer(data, i: int, r: ConfigReader, where: str) -> Optional[LayerConfig]:
    if not isinstance(data, dict):
        r.problem(f"layers[{i}] must be an object")
        return None
    n0 = len(r.problems)
    lr = ConfigReader(data, f"{where}.layers[{i}]")
    lr.problems = r.problems
    kind = lr.string("type", choices=(PARALLEL,))
    weights_of = lr.integer("weights_of", minimum=0) if data.get("weights_of") is not None else None
    m = _sub(lr, "mixer", lr.where)
    mixer = None
    if m is not None and kind == PARALLEL:
        left, right = _left(m, r, i), _right(m, r, i)
        ls, rs = m.number("left_scale", default=1.0, positive=False), m.number("right_scale", default=1.0, positive=False)
        if None not in (left, right, ls, rs):
            mixer = ParallelMixerConfig(left, right, ls, rs)
    mlp = _mlp(lr, r, i) if data.get("mlp") is not None else None
    if len(r.problems) > n0 or kind is None or mixer is None:
        return None
    return LayerConfig(kind, mixer, mlp, weights_of)


def weight_owner(layers, i: int) -> Optional[int]:
    """The layer whose tensors layer i uses (None: its `weights_of` leads nowhere)."""
    seen = set()
    while layers[i].weights_of is not None:
        if i in seen or not 0 <= layers[i].weights_of < len(layers):
            return None
        seen.add(i)
        i = layers[i].weights_of
    return i


@dataclass(frozen=True)
class KugisunConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int            # 0: the key is absent, one plain stream without coefficients
    layers: Tuple[LayerConfig, ...]
    max_positions: int
    raw: dict

    architecture = "Kugisun"

    @classmethod
    def from_dict(cls, data: dict, where: str = "config.json") -> "KugisunConfig":
        r = ConfigReader(data, where)
        vocab, width = r.integer("vocab"), r.integer("width")
        norm = _sub(r, "norm", where)
        eps = norm.number("eps") if norm is not None else None
        streams = r.integer("streams", default=0, minimum=0)
        max_positions = r.integer("max_positions")
        layers = r.raw("layers")
        parsed = []
        if not isinstance(layers, list) or not layers:
            r.problem("'layers' must be a non-empty list")
        else:
            parsed = [_layer(d, i, r, where) for i, d in enumerate(layers)]
        if parsed and None not in parsed:
            for i, layer in enumerate(parsed):
                j = weight_owner(parsed, i)
                if j is None:
                    r.problem(f"layers[{i}].weights_of {layer.weights_of} leads to no layer with tensors")
                elif (layer.type, layer.mixer, layer.mlp) != (parsed[j].type, parsed[j].mixer, parsed[j].mlp):
                    r.problem(f"layers[{i}] uses the tensors of layer {j} and differs from it")
        if streams is not None:
            r.check(streams <= 16, f"streams {streams}: at most 16")
        r.finish()
        return cls(vocab, width, eps, streams, tuple(parsed), max_positions, dict(data))

    def to_dict(self) -> dict:
        return dict(self.raw)

    @staticmethod
    def fill_from_tensor_shapes(data: dict, shapes: dict) -> dict:
        """`data` with `max_positions` from the shape of the folder's table of positions, if the file does not name it."""
        if data.get("max_positions") is None and len(shapes.get("pos", ())) == 2:
            return {**data, "max_positions": int(shapes["pos"][0])}
        return data
