"""Typed configuration of Sokipel, read from the keys of its own config.json.

The file is nested: ``vocab``, ``width``, ``norm`` (eps), ``embedding`` (scale), ``residual_mult``, ``canon`` (taps of the
convolution in front of every mixer), ``logit_softcap`` and ``layers``, a list with one entry per layer: the mixer's ``type``
(``attention``, ``delta`` or ``parallel``), its sizes and constants (``mixer``) and the feed-forward (``mlp``: ``kind`` ``moe``,
or null for none).  Nothing is assumed about the number or the order of the layers, and every size and constant comes from
the file.  The design gives no limit on positions; ``DEFAULT_MAX_POSITIONS`` bounds what an engine may be built for.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..errors import ConfigError
from . import fields as F
from .puledra import _section

DEFAULT_MAX_POSITIONS = 1 << 20


@dataclass(frozen=True)
class Rotation:
    dims: int               # leading dims of every q and k head that rotate
    base: float
    banded: tuple | None = None      # (factor, low, high, original) or None
    linear: float | None = None      # every frequency is divided by it, or None


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int                # query/key dims per head
    vdim: int               # value dims per head
    scale: float
    rot: Rotation | None
    chunk: int              # a position sees the earlier positions of its own chunk of so many (0: all earlier ones)


@dataclass(frozen=True)
class DeltaRule:
    heads: int              # value heads
    kv_heads: int           # query/key heads
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class Parallel:
    left: Attention
    right: DeltaRule
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class ExpertMlp:
    ff: int
    limit: float            # of the clamped activation
    experts: int
    top: int


@dataclass(frozen=True)
class SokipelLayer:
    mixer: object           # Attention, DeltaRule or Parallel
    mlp: ExpertMlp | None


def _heads(m, where):
    heads, kv = F.get_int(m, "heads", minimum=1), F.get_int(m, "kv_heads", minimum=1)
    if heads % kv:
        raise ConfigError(f"{where}.heads {heads} is not a multiple of kv_heads {kv}")
    return {"heads": heads, "kv_heads": kv, "dim": F.get_int(m, "dim", minimum=1), "vdim": F.get_int(m, "vdim", minimum=1)}


def _rotation(m, dim, banded, where):
    rot = _section(m, "rot", optional=True)
    if rot is None or F.get_int(rot, "dims", minimum=0) == 0:
        return None
    dims = F.get_int(rot, "dims")
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}.rot.dims must be even and at most dim {dim}, got {dims}")
    base, sc = F.get_float(rot, "base"), _section(rot, "scaling", optional=True)
    if sc is None:
        return Rotation(dims, base)
    factor = F.get_float(sc, "factor")
    if factor <= 0:
        raise ConfigError(f"{where}.rot.scaling.factor must be positive, got {factor}")
    if not banded:
        return Rotation(dims, base, linear=factor)
    low, high, original = (F.get_float(sc, k) for k in ("low", "high", "original"))
    if min(low, high, original) <= 0 or high < low:
        raise ConfigError(f"{where}.rot.scaling: low, high and original must be positive, and high at least low")
    return Rotation(dims, base, banded=(factor, low, high, original))


def _attention(m, where, banded, masked):
    sizes = _heads(m, where)
    mask = _section(m, "mask", optional=True) if masked else None
    return Attention(**sizes, scale=F.get_float(m, "scale"), rot=_rotation(m, sizes["dim"], banded, where),
                     chunk=F.get_int(mask, "size", minimum=1) if mask is not None else 0)


def _delta(m, where):
    return DeltaRule(**_heads(m, where), taps=F.get_int(m, "conv", minimum=1))


def _mixer(kind, m, where):
    if kind == "attention":
        return _attention(m, where, banded=True, masked=True)
    if kind == "delta":
        return _delta(m, where)
    if kind == "parallel":
        return Parallel(_attention(_section(m, "left"), where + ".left", banded=False, masked=False),
                        _delta(_section(m, "right"), where + ".right"), F.get_float(m, "left_scale"), F.get_float(m, "right_scale"))
    raise ConfigError(f"{where}: unknown layer type {kind!r} (known: attention, delta, parallel)")


def _mlp(f, where):
    kind = F.get_str(f, "kind")
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind {kind!r} (known: moe)")
    e, r = _section(f, "expert"), _section(f, "router")
    out = ExpertMlp(ff=F.get_int(e, "ff", minimum=1), limit=F.get_float(e, "limit"), experts=F.get_int(r, "experts", minimum=1),
                    top=F.get_int(r, "top", minimum=1))
    if out.limit <= 0:
        raise ConfigError(f"{where}.expert.limit must be positive, got {out.limit}")
    if out.top > out.experts:
        raise ConfigError(f"{where}.router.top {out.top} exceeds the {out.experts} experts")
    return out


@dataclass(frozen=True)
class SokipelConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    residual_mult: float
    canon_taps: int
    softcap: float          # logits <- softcap tanh(logits / softcap)
    layers: tuple
    architecture: str = "Sokipel"

    @classmethod
    def from_dict(cls, d: dict) -> "SokipelConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a non-empty list")
        out = []
        for i, entry in enumerate(layers):
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            f = _section(entry, "mlp", optional=True)
            out.append(SokipelLayer(_mixer(F.get_str(entry, "type"), _section(entry, "mixer"), f"layers[{i}].mixer"),
                                    _mlp(f, f"layers[{i}].mlp") if f is not None else None))
        softcap = F.get_float(d, "logit_softcap")
        if softcap <= 0:
            raise ConfigError(f"config field 'logit_softcap' must be positive, got {softcap}")
        return cls(vocab=F.get_int(d, "vocab", minimum=1), width=F.get_int(d, "width", minimum=1),
                   eps=F.get_float(_section(d, "norm"), "eps"), embed_scale=F.get_float(_section(d, "embedding"), "scale"),
                   residual_mult=F.get_float(d, "residual_mult"), canon_taps=F.get_int(_section(d, "canon"), "taps", minimum=1),
                   softcap=softcap, layers=tuple(out))
