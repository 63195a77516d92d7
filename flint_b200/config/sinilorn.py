"""Typed configuration of Sinilorn, read from the keys of its own config.json.

The file is nested: ``vocab``, ``width``, ``streams``, ``norm`` (eps), ``logit_scale`` and ``layers`` (a list with one
entry per layer: the mixer's ``type`` (``latent_attention`` or ``rglru``), the mixer's sizes and constants (``mixer``) and
the feed-forward (``mlp``: ``kind`` ``dense`` or ``moe``, or null for none)).  Nothing is assumed about the number or the
order of the layers, and every size and constant comes from the file.  The design gives no limit on positions;
``DEFAULT_MAX_POSITIONS`` bounds what an engine may be built for.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..errors import ConfigError
from . import fields as F
from .puledra import _section

DEFAULT_MAX_POSITIONS = 1 << 20


@dataclass(frozen=True)
class Rotation:
    base: float
    yarn: tuple | None      # (factor, original, fast, slow) or None


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int                # unrotated query/key dims per head
    rot_dim: int            # rotated dims per head; the rotated key part is shared by all heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotation | None
    window: int             # 0: every earlier position is seen
    kv_from: int | None     # the layer whose latent rows this one reads, or None for its own


@dataclass(frozen=True)
class RecurrentUnit:
    width: int
    blocks: int
    taps: int


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class ExpertMlp:
    ff: int
    limit: float            # of the clamped activation
    experts: int
    identity: int           # router outputs whose expert hands its input on
    top: int


@dataclass(frozen=True)
class SinilornLayer:
    mixer: object           # LatentAttention or RecurrentUnit
    mlp: object             # DenseMlp, ExpertMlp or None


def _rotation(m, rot_dim, where):
    rot = _section(m, "rot", optional=True)
    if rot_dim == 0:
        return None
    if rot is None:
        raise ConfigError(f"missing config field {where + '.rot'!r}")
    if rot_dim % 2 or F.get_int(rot, "dims", rot_dim) != rot_dim:
        raise ConfigError(f"{where}.rot.dims must equal rot_dim {rot_dim} and be even, got {rot.get('dims')}")
    sc = _section(rot, "scaling", optional=True)
    yarn = None
    if sc is not None:
        yarn = (F.get_float(sc, "factor"), F.get_float(sc, "original"), F.get_float(sc, "fast"), F.get_float(sc, "slow"))
        if min(yarn) <= 0:
            raise ConfigError(f"{where}.rot.scaling: factor, original, fast and slow must be positive")
    return Rotation(F.get_float(rot, "base"), yarn)


def _mixer(kind, m, where):
    if kind == "rglru":
        u = RecurrentUnit(F.get_int(m, "width", minimum=1), F.get_int(m, "blocks", minimum=1), F.get_int(m, "conv", minimum=1))
        if u.width % u.blocks:
            raise ConfigError(f"{where}.width {u.width} is not a multiple of blocks {u.blocks}")
        return u
    if kind == "latent_attention":
        rot_dim = F.get_int(m, "rot_dim", minimum=0)
        mask = _section(m, "mask", optional=True)
        return LatentAttention(
            heads=F.get_int(m, "heads", minimum=1), dim=F.get_int(m, "dim", minimum=0 if rot_dim else 1), rot_dim=rot_dim,
            vdim=F.get_int(m, "vdim", minimum=1), q_rank=F.get_int(m, "q_rank", minimum=1),
            kv_rank=F.get_int(m, "kv_rank", minimum=1), scale=F.get_float(m, "scale"), rot=_rotation(m, rot_dim, where),
            window=F.get_int(mask, "size", minimum=1) if mask is not None else 0,
            kv_from=F.get_int(m, "kv_from", None, minimum=0))
    raise ConfigError(f"{where}: unknown layer type {kind!r} (known: latent_attention, rglru)")


def _mlp(f, where):
    kind = F.get_str(f, "kind")
    if kind == "dense":
        return DenseMlp(F.get_int(f, "ff", minimum=1))
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind {kind!r} (known: dense, moe)")
    e, r = _section(f, "expert"), _section(f, "router")
    out = ExpertMlp(ff=F.get_int(e, "ff", minimum=1), limit=F.get_float(e, "limit"), experts=F.get_int(r, "experts", minimum=1),
                    identity=F.get_int(r, "identity", 0, minimum=0), top=F.get_int(r, "top", minimum=1))
    if out.limit <= 0:
        raise ConfigError(f"{where}.expert.limit must be positive, got {out.limit}")
    if out.top > out.experts + out.identity:
        raise ConfigError(f"{where}.router.top {out.top} exceeds the {out.experts} + {out.identity} experts")
    return out


@dataclass(frozen=True)
class SinilornConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    logit_scale: float
    layers: tuple
    architecture: str = "Sinilorn"

    @classmethod
    def from_dict(cls, d: dict) -> "SinilornConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a non-empty list")
        out = []
        for i, entry in enumerate(layers):
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            f = _section(entry, "mlp", optional=True)
            out.append(SinilornLayer(_mixer(F.get_str(entry, "type"), _section(entry, "mixer"), f"layers[{i}].mixer"),
                                     _mlp(f, f"layers[{i}].mlp") if f is not None else None))
        for i, layer in enumerate(out):
            m = layer.mixer
            if not isinstance(m, LatentAttention) or m.kv_from is None:
                continue
            src = out[m.kv_from].mixer if m.kv_from < i else None
            if not isinstance(src, LatentAttention) or src.kv_from is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from {m.kv_from} must name an earlier latent_attention layer with "
                                  f"latent rows of its own")
            if (src.kv_rank, src.rot_dim, src.rot) != (m.kv_rank, m.rot_dim, m.rot):
                raise ConfigError(f"layers[{i}].mixer.kv_from {m.kv_from}: latent size, rot_dim and rotation must be equal")
        return cls(vocab=F.get_int(d, "vocab", minimum=1), width=F.get_int(d, "width", minimum=1),
                   eps=F.get_float(_section(d, "norm"), "eps"), streams=F.get_int(d, "streams", minimum=1),
                   logit_scale=F.get_float(d, "logit_scale", 1.0), layers=tuple(out))
