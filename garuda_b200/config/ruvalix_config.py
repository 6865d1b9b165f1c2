"""Typed configuration of the Ruvalix design, read from its config.json.

Keys: ``architecture`` ("Ruvalix"), ``vocab``, ``width``, ``norm.eps``, ``layers``
(a list; each entry has ``type`` = ``attention`` | ``mlstm``, the mixer's sizes
under ``mixer``, its feed-forward under ``mlp`` or null), ``loop`` (``start``,
``stop``, ``times``; optional), ``max_positions`` (optional: the longest
sequence; the design itself has no limit).

``attention``: ``heads``, ``kv_heads``, ``dim`` (of one map), ``vdim``, ``scale``,
``diff``, ``mask.size`` (optional: every earlier position is seen), ``rot.base`` and
``rot.dims`` (optional: not rotated), ``rot.scaling`` (optional: ``factor``, ``original``,
``fast``, ``slow``).
``mlstm``: ``heads``, ``dim``, ``vdim``, ``gate_cap``.
``mlp``: ``kind`` = ``moe``; ``expert.ff``, ``router.experts``, ``router.top``, ``router.identity``
(optional: none), ``router.groups.count`` and ``.keep`` (optional: one group), ``shared.ff``
(optional: no shared expert).
Every size and constant of a model comes from here; a key that is missing
where the design needs it is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple

from .kavenex_config import _get
from .model_config import ConfigError

MIXER_TYPES = ("attention", "mlstm")
DEFAULT_MAX_POSITIONS = 32768


@dataclass(frozen=True)
class YarnConfig:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                     # query/key channels of one map
    vdim: int
    scale: float
    diff: float
    window: Optional[int]
    rot_base: Optional[float]
    rot_dims: int
    rot_scaling: Optional[YarnConfig]


@dataclass(frozen=True)
class MlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    ff: int
    identity: int
    groups: Optional[Tuple[int, int]]        # (count, keep)
    shared_ff: Optional[int]


@dataclass(frozen=True)
class RuvalixLayer:
    type: str
    mixer: object
    mlp: Optional[MoeConfig]


def _read_attention(m, w):
    heads, kv_heads = _get(m, "heads", w, int, 1), _get(m, "kv_heads", w, int, 1)
    dim, vdim = _get(m, "dim", w, int, 1), _get(m, "vdim", w, int, 1)
    if heads % kv_heads:
        raise ConfigError(f"config.json: '{w}heads' = {heads} is not a multiple of '{w}kv_heads' = {kv_heads}")
    window = _get(m["mask"], "size", w + "mask.", int, 1) if m.get("mask") is not None else None
    base, dims, scaling = None, 0, None
    if m.get("rot") is not None:
        r, wr = m["rot"], w + "rot."
        base, dims = _get(r, "base", wr, float, 0.0), _get(r, "dims", wr, int, 2)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: '{wr}dims' = {dims} must be even and at most '{w}dim' = {dim}")
        if r.get("scaling") is not None:
            s, ws = r["scaling"], wr + "scaling."
            scaling = YarnConfig(*(_get(s, key, ws, float, 0.0) for key in ("factor", "original", "fast", "slow")))
            if base == 1.0:
                raise ConfigError(f"config.json: '{wr}base' = 1 has no wavelengths to scale")
    return DifferentialAttentionConfig(heads, kv_heads, dim, vdim, _get(m, "scale", w, float), _get(m, "diff", w, float), window,
                                       base, dims, scaling)


def _read_mlstm(m, w):
    return MlstmConfig(*(_get(m, key, w, int, 1) for key in ("heads", "dim", "vdim")), _get(m, "gate_cap", w, float, 0.0))


def _read_mlp(f, w):
    kind = _get(f, "kind", w)
    if kind != "moe":
        raise ConfigError(f"config.json: '{w}kind' = {kind!r}: this design's feed-forward is 'moe'")
    r, wr = _get(f, "router", w), w + "router."
    experts, top = _get(r, "experts", wr, int, 1), _get(r, "top", wr, int, 1)
    identity = _get(r, "identity", wr, int, 0) if r.get("identity") is not None else 0
    choices, groups = experts + identity, None
    if r.get("groups") is not None:
        count, keep = (_get(r["groups"], key, wr + "groups.", int, 1) for key in ("count", "keep"))
        if choices % count or keep > count:
            raise ConfigError(f"config.json: '{wr}groups' = {count}, {keep}: {choices} choices must split into equal groups of which some are kept")
        groups = (count, keep)
    within = choices if groups is None else choices // groups[0] * groups[1]
    if top > within:
        raise ConfigError(f"config.json: '{wr}top' = {top} is more than the {within} that can be chosen")
    shared = _get(f["shared"], "ff", w + "shared.", int, 1) if f.get("shared") is not None else None
    return MoeConfig(experts, top, _get(_get(f, "expert", w), "ff", w + "expert.", int, 1), identity, groups, shared)


@dataclass(frozen=True)
class RuvalixConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[RuvalixLayer, ...]
    loop: Optional[Tuple[int, int, int]]     # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()
    raw: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, d: dict) -> "RuvalixConfig":
        vocab, width = _get(d, "vocab", "", int, 1), _get(d, "width", "", int, 1)
        eps = _get(d.get("norm"), "eps", "norm.", float, 0.0)
        entries = _get(d, "layers", "")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, e in enumerate(entries):
            w = f"layers[{i}]."
            kind = _get(e, "type", w)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{w}type' = {kind!r} is not a mixer of this design {MIXER_TYPES}")
            read = _read_attention if kind == "attention" else _read_mlstm
            mixer = read(_get(e, "mixer", w), w + "mixer.")
            layers.append(RuvalixLayer(kind, mixer, _read_mlp(e["mlp"], w + "mlp.") if e.get("mlp") is not None else None))
        loop = None
        if d.get("loop") is not None:
            start, stop, times = (_get(d["loop"], key, "loop.", int, low) for key, low in (("start", 0), ("stop", 1), ("times", 1)))
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: 'loop' runs layers {start} to {stop - 1} of {len(layers)}")
            loop = (start, stop, times)
        eos = d.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        return cls(architecture=d.get("architecture", "Ruvalix"), vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                   loop=loop, max_positions=int(d.get("max_positions") or DEFAULT_MAX_POSITIONS), eos_token_ids=eos, raw=dict(d))

    def to_dict(self) -> dict:
        return dict(self.raw)
