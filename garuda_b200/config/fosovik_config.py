"""Typed configuration of the Fosovik design, read from its config.json.

Keys: ``architecture`` ("Fosovik"), ``vocab``, ``width``, ``embedding.scale``,
``norm.eps``, ``layers`` (a list; each entry has ``type`` = ``attention`` |
``mamba2``, the mixer's sizes under ``mixer``, its feed-forward under ``mlp`` or
null), ``max_positions`` (optional: the longest sequence; the design itself has
no limit).

``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
``q_temp.coef`` and ``q_temp.every`` (optional: queries are not scaled by their
position), ``kv_from`` (optional: the earlier layer whose keys and values are
read).
``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps),
``norm_groups``.
``mlp``: ``kind`` = ``dense`` (``ff``, ``limit``) | ``moe`` (``expert.ff``,
``router.experts``, ``router.top``).
Every size and constant of a model comes from here; a key that is missing
where the design needs it is an error that names it.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple

from .kavenex_config import _get
from .model_config import ConfigError

MIXER_TYPES = ("attention", "mamba2")
DEFAULT_MAX_POSITIONS = 32768


@dataclass(frozen=True)
class SharedKvAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[Tuple[float, int]]      # (coef, every)
    kv_from: Optional[int]


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class MlpConfig:
    kind: str                    # "dense" | "moe"
    ff: int
    limit: float = 0.0           # dense
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class FosovikLayer:
    type: str
    mixer: object
    mlp: Optional[MlpConfig]


def _read_mixer(kind, m, wm):
    heads, vdim = _get(m, "heads", wm, int, 1), _get(m, "vdim", wm, int, 1)
    if kind == "mamba2":
        state, groups, taps = (_get(m, key, wm, int, 1) for key in ("state", "groups", "conv"))
        norm_groups = _get(m, "norm_groups", wm, int, 1)
        if heads % groups:
            raise ConfigError(f"config.json: '{wm}heads' = {heads} is not a multiple of '{wm}groups' = {groups}")
        if heads * vdim % norm_groups:
            raise ConfigError(f"config.json: the {heads * vdim} channels of '{wm}' do not split into "
                              f"'{wm}norm_groups' = {norm_groups} equal parts")
        if taps > 16:
            raise ConfigError(f"config.json: '{wm}conv' = {taps}: at most 16 taps")
        return Mamba2Config(heads, vdim, state, groups, taps, norm_groups)
    kv_heads = _get(m, "kv_heads", wm, int, 1)
    if heads % kv_heads:
        raise ConfigError(f"config.json: '{wm}heads' = {heads} is not a multiple of '{wm}kv_heads' = {kv_heads}")
    temp = None
    if m.get("q_temp") is not None:
        temp = (_get(m["q_temp"], "coef", wm + "q_temp.", float), _get(m["q_temp"], "every", wm + "q_temp.", int, 1))
    source = _get(m, "kv_from", wm, int, 0) if m.get("kv_from") is not None else None
    return SharedKvAttentionConfig(heads, kv_heads, _get(m, "dim", wm, int, 1), vdim, _get(m, "scale", wm, float, 0.0), temp, source)


def _read_mlp(f, w):
    kind = _get(f, "kind", w)
    if kind == "dense":
        return MlpConfig("dense", _get(f, "ff", w, int, 1), limit=_get(f, "limit", w, float, 0.0))
    if kind == "moe":
        router = _get(f, "router", w)
        experts, top = _get(router, "experts", w + "router.", int, 1), _get(router, "top", w + "router.", int, 1)
        if top > experts:
            raise ConfigError(f"config.json: '{w}router.top' = {top} is more than '{w}router.experts' = {experts}")
        return MlpConfig("moe", _get(_get(f, "expert", w), "ff", w + "expert.", int, 1), experts=experts, top=top)
    raise ConfigError(f"config.json: '{w}kind' = {kind!r}: this design's feed-forwards are 'dense' and 'moe'")


@dataclass(frozen=True)
class FosovikConfig:
    architecture: str
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    layers: Tuple[FosovikLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: tuple = ()
    raw: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, d: dict) -> "FosovikConfig":
        vocab = _get(d, "vocab", "", int, 1)
        width = _get(d, "width", "", int, 1)
        scale = _get(d.get("embedding"), "scale", "embedding.", float)
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
            mixer = _read_mixer(kind, _get(e, "mixer", w), w + "mixer.")
            if kind == "attention" and mixer.kv_from is not None:
                src = layers[mixer.kv_from] if mixer.kv_from < i else None
                if src is None or src.type != "attention" or src.mixer.kv_from is not None:
                    raise ConfigError(f"config.json: '{w}mixer.kv_from' = {mixer.kv_from} must name an earlier attention layer "
                                      "with keys and values of its own")
                if (src.mixer.kv_heads, src.mixer.dim, src.mixer.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ConfigError(f"config.json: '{w}mixer' reads the keys and values of layer {mixer.kv_from} "
                                      "but its key/value heads have other sizes")
            mlp = _read_mlp(e["mlp"], w + "mlp.") if e.get("mlp") is not None else None
            layers.append(FosovikLayer(kind, mixer, mlp))
        eos = d.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        return cls(architecture=d.get("architecture", "Fosovik"), vocab=vocab, width=width, embedding_scale=scale, eps=eps,
                   layers=tuple(layers), max_positions=int(d.get("max_positions") or DEFAULT_MAX_POSITIONS),
                   eos_token_ids=eos, raw=dict(d))

    def to_dict(self) -> dict:
        return dict(self.raw)
