"""Typed configuration of the Pagulix decoder, read from config.json.

What config.json holds (sizes and constants come from nowhere else):

    {"architecture": "Pagulix", "vocab": V, "width": D, "streams": S, "residual_mult": m, "logit_softcap": c,
     "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot": {"base", "dims"},
                           "mask": {"size"} (optional)},
                 "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"} (optional)}},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "v_mix" (optional),
                           "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"} (optional)}}, "mlp": ...},
                {"type": "delta", "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}, "mlp": ...},
                ...]}

Sizes and constants have no defaults: a missing key is an error that names it.  Optional are only the things a layer may
lack: `mask` (every earlier position is visible), `scaling` (plain frequencies), `v_mix` (the layer's own values), `shared`,
`mlp`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .lulisun_config import _float, _get, _int
from .model_config import ConfigError

ARCHITECTURE = "Pagulix"


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                 # unrotated channels of a query / key head
    rot_dim: int             # rotated ones, whose key part all heads share
    vdim: int
    kv_rank: int
    scale: float             # on the scores
    rot_base: float
    window: int | None       # a query sees itself and the window - 1 positions before it (None: all)


@dataclass(frozen=True)
class WaveScalingConfig:
    """Frequencies by how often a channel's wave turns over the original context: more than `high` times as they are, fewer
    than `low` times divided by `factor`, blended between."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int            # rotated channels of a head (the first ones)
    scaling: WaveScalingConfig | None
    v_mix: bool              # values are blended with those of the first layer that says so


@dataclass(frozen=True)
class DeltaRuleConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    top: int
    shared_ff: int | None


@dataclass(frozen=True)
class PagulixLayerConfig:
    kind: str                # "latent_attention" | "attention" | "delta"
    mixer: Any
    mlp: MoeConfig | None
    raw: Any = None


def _shared_heads(m: Mapping, w: str) -> tuple:
    heads, kv = _int(m, "heads", w), _int(m, "kv_heads", w)
    if heads % kv:
        raise ConfigError(f"config.json: {w}: {heads} heads are not a multiple of {kv} kv heads")
    return heads, kv


def _positive(d: Mapping, key: str, w: str) -> float:
    v = _float(d, key, w)
    if not v > 0:
        raise ConfigError(f"config.json: {w}.{key} must be positive, found {v!r}")
    return v


def _rotated(rot: Mapping, w: str, most: int) -> int:
    dims = _int(rot, "dims", w)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {w}.dims must be even and at most {most}, found {dims}")
    return dims


def _latent(m: Mapping, w: str) -> LatentAttentionConfig:
    rot, rot_dim = _get(m, "rot", w), _int(m, "rot_dim", w)
    if _rotated(rot, w + ".rot", rot_dim) != rot_dim:
        raise ConfigError(f"config.json: {w}.rot.dims must be the size of the rotated part, {rot_dim}")
    window = None if m.get("mask") is None else _int(m["mask"], "size", w + ".mask")
    return LatentAttentionConfig(heads=_int(m, "heads", w), dim=_int(m, "dim", w), rot_dim=rot_dim, vdim=_int(m, "vdim", w),
                                 kv_rank=_int(m, "kv_rank", w), scale=_float(m, "scale", w),
                                 rot_base=_positive(rot, "base", w + ".rot"), window=window)


def _attention(m: Mapping, w: str) -> AttentionConfig:
    heads, kv = _shared_heads(m, w)
    rot, rw, dim = _get(m, "rot", w), w + ".rot", _int(m, "dim", w)
    scaling = None
    if rot.get("scaling") is not None:
        s, sw = rot["scaling"], rw + ".scaling"
        scaling = WaveScalingConfig(factor=_positive(s, "factor", sw), low=_float(s, "low", sw), high=_float(s, "high", sw),
                                    original=_positive(s, "original", sw))
        if not scaling.high > scaling.low:
            raise ConfigError(f"config.json: {sw}.high must be above low, found {scaling.high} and {scaling.low}")
    mix = m.get("v_mix") or False
    if not isinstance(mix, bool):
        raise ConfigError(f"config.json: {w}.v_mix must be true or false, found {mix!r}")
    return AttentionConfig(heads=heads, kv_heads=kv, dim=dim, vdim=_int(m, "vdim", w), scale=_float(m, "scale", w),
                           rot_base=_positive(rot, "base", rw), rot_dims=_rotated(rot, rw, dim), scaling=scaling, v_mix=mix)


def _delta(m: Mapping, w: str) -> DeltaRuleConfig:
    heads, kv = _shared_heads(m, w)
    return DeltaRuleConfig(heads=heads, kv_heads=kv, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w), conv=_int(m, "conv", w))


_MIXERS = {"latent_attention": _latent, "attention": _attention, "delta": _delta}


def _feed_forward(f: Mapping | None, w: str) -> MoeConfig | None:
    if f is None:
        return None
    kind = _get(f, "kind", w)
    if kind != "moe":
        raise ConfigError(f"config.json: {w}.kind {kind!r} is not a feed-forward of this design (have: 'moe')")
    r, rw = _get(f, "router", w), w + ".router"
    shared = None if f.get("shared") is None else _int(f["shared"], "ff", w + ".shared")
    m = MoeConfig(ff=_int(_get(f, "expert", w), "ff", w + ".expert"), experts=_int(r, "experts", rw), top=_int(r, "top", rw),
                  shared_ff=shared)
    if m.top > m.experts:
        raise ConfigError(f"config.json: {rw}: {m.experts} experts cannot give {m.top} choices")
    return m


@dataclass(frozen=True)
class PagulixConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    streams: int             # parallel copies of the hidden stream
    residual_mult: float     # on what a sublayer adds to them
    logit_softcap: float
    norm_eps: float
    layers: tuple
    raw: Any = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "PagulixConfig":
        entries = _get(d, "layers", "the model")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers, first = [], None
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            kind, m, mw = _get(entry, "type", where), _get(entry, "mixer", where), where + ".mixer"
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (have: {', '.join(map(repr, _MIXERS))})")
            mixer = _MIXERS[kind](m, mw)
            if kind == "attention" and mixer.v_mix:
                first = first or (i, mixer)
                if (mixer.kv_heads, mixer.vdim) != (first[1].kv_heads, first[1].vdim):
                    raise ConfigError(f"config.json: {mw}: values of {mixer.kv_heads} x {mixer.vdim} cannot be blended with those of "
                                      f"layer {first[0]}, {first[1].kv_heads} x {first[1].vdim}")
            layers.append(PagulixLayerConfig(kind, mixer, _feed_forward(entry.get("mlp"), where + ".mlp"), raw=entry))
        return cls(architecture=ARCHITECTURE, vocab_size=_int(d, "vocab", "the model"), hidden_size=_int(d, "width", "the model"),
                   streams=_int(d, "streams", "the model"), residual_mult=_float(d, "residual_mult", "the model"),
                   logit_softcap=_positive(d, "logit_softcap", "the model"),
                   norm_eps=_positive(_get(d, "norm", "the model"), "eps", "norm"), layers=tuple(layers), raw=dict(d))

    def to_dict(self) -> dict:
        """The config.json form."""
        layers = []
        for L in self.layers:
            m, f = L.mixer, L.mlp
            if L.kind == "latent_attention":
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                         "scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dim}}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window}
            elif L.kind == "attention":
                rot = {"base": m.rot_base, "dims": m.rot_dims}
                if m.scaling is not None:
                    s = m.scaling
                    rot["scaling"] = {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot,
                         "v_mix": m.v_mix}
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            mlp = None
            if f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff is not None:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": L.kind, "mixer": mixer, "mlp": mlp})
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap, "norm": {"eps": self.norm_eps},
                "layers": layers}
