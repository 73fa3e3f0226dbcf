"""Typed configuration of the Gatarax decoder, read from config.json.

What config.json holds (sizes and constants come from nowhere else):

    {"architecture": "Gatarax", "vocab": V, "width": D, "norm": {"eps": e}, "canon": {"taps": K},
     "embedding": {"scale": s}, "logit_scale": c,
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "conv", "mask": {"size"} (optional)},
                           "right": {"heads", "kv_heads", "dim", "vdim", "conv",
                                     "decay_rank" (optional), "gate_rank" (optional)}},
                 "mlp": null | {"kind": "dense", "ff"}
                            | {"kind": "moe", "expert": {"ff"},
                               "router": {"experts", "top", "groups": {"count", "keep"} (optional)}}},
                {"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [one per head]}, "mlp": ...},
                ...]}

Sizes and constants have no defaults: a missing key is an error that names it.  Optional are only the things a layer may
lack: `mask` (every earlier position is visible), `groups` (the experts are one group), `mlp`.  The ranks of a delta
rule's two low-rank maps are the sizes config.json may leave to the weights: without `decay_rank` / `gate_rank` they are the
number of rows of the tensors `l<i>.mix.right.a1` / `l<i>.mix.right.g1`, which the caller hands over as `shapes`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .lulisun_config import _float, _get, _int
from .model_config import ConfigError

ARCHITECTURE = "Gatarax"


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                 # size of a query / key head
    vdim: int                # size of a value head
    scale: float             # on the scores
    conv: int                # taps of the short convolutions behind the projections
    window: int | None       # a query sees itself and the window - 1 positions before it (None: all)


@dataclass(frozen=True)
class DeltaRuleConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowAttentionConfig
    right: DeltaRuleConfig


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple             # one number per head


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    top: int
    groups: int              # equal groups of neighbouring experts
    keep: int                # groups whose experts can be chosen


@dataclass(frozen=True)
class GataraxLayerConfig:
    kind: str                # "parallel" | "lightning"
    mixer: Any
    mlp: Any                 # DenseMlpConfig | MoeConfig | None
    raw: Any = None


def _shared_heads(m: Mapping, w: str) -> tuple:
    heads, kv = _int(m, "heads", w), _int(m, "kv_heads", w)
    if heads % kv:
        raise ConfigError(f"config.json: {w}: {heads} heads are not a multiple of {kv} kv heads")
    return heads, kv


def _rank(m: Mapping, key: str, w: str, tensor: str, shapes) -> int:
    if m.get(key) is not None:
        return _int(m, key, w)
    if shapes is not None and len(shapes.get(tensor, ())) == 2:
        return int(shapes[tensor][0])
    raise ConfigError(f"config.json: {w}.{key} is missing, and so is the tensor {tensor} whose rows give it")


def _left(m: Mapping, w: str) -> WindowAttentionConfig:
    heads, kv = _shared_heads(m, w)
    window = None if m.get("mask") is None else _int(m["mask"], "size", w + ".mask")
    return WindowAttentionConfig(heads=heads, kv_heads=kv, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w),
                                 scale=_float(m, "scale", w), conv=_int(m, "conv", w), window=window)


def _right(m: Mapping, w: str, prefix: str, shapes) -> DeltaRuleConfig:
    heads, kv = _shared_heads(m, w)
    return DeltaRuleConfig(heads=heads, kv_heads=kv, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w), conv=_int(m, "conv", w),
                           decay_rank=_rank(m, "decay_rank", w, prefix + "a1", shapes),
                           gate_rank=_rank(m, "gate_rank", w, prefix + "g1", shapes))


def _lightning(m: Mapping, w: str) -> LightningConfig:
    heads, decay = _int(m, "heads", w), _get(m, "decay", w)
    if not isinstance(decay, (list, tuple)) or len(decay) != heads:
        raise ConfigError(f"config.json: {w}.decay must list one number for each of the {heads} heads, found {decay!r}")
    if any(isinstance(c, bool) or not isinstance(c, (int, float)) for c in decay):
        raise ConfigError(f"config.json: {w}.decay must be numbers, found {decay!r}")
    return LightningConfig(heads=heads, dim=_int(m, "dim", w), vdim=_int(m, "vdim", w), decay=tuple(float(c) for c in decay))


def _feed_forward(f: Mapping | None, w: str):
    if f is None:
        return None
    kind = _get(f, "kind", w)
    if kind == "dense":
        return DenseMlpConfig(ff=_int(f, "ff", w))
    if kind != "moe":
        raise ConfigError(f"config.json: {w}.kind {kind!r} is not a feed-forward of this design (have: 'dense', 'moe')")
    r, rw = _get(f, "router", w), w + ".router"
    count, keep = 1, 1
    if r.get("groups") is not None:
        count, keep = _int(r["groups"], "count", rw + ".groups"), _int(r["groups"], "keep", rw + ".groups")
    m = MoeConfig(ff=_int(_get(f, "expert", w), "ff", w + ".expert"), experts=_int(r, "experts", rw), top=_int(r, "top", rw),
                  groups=count, keep=keep)
    if m.experts % m.groups or m.keep > m.groups:
        raise ConfigError(f"config.json: {rw}: {m.experts} experts do not form {m.groups} equal groups of which {m.keep} are kept")
    if m.top > m.keep * (m.experts // m.groups):
        raise ConfigError(f"config.json: {rw}: {m.keep} groups of {m.experts // m.groups} experts cannot give {m.top} choices")
    return m


@dataclass(frozen=True)
class GataraxConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    taps: int                # of the convolutions in front of mixer and feed-forward
    embedding_scale: float
    logit_scale: float
    layers: tuple
    raw: Any = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], shapes: Mapping[str, tuple] | None = None) -> "GataraxConfig":
        entries = _get(d, "layers", "the model")
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            kind, m, mw = _get(entry, "type", where), _get(entry, "mixer", where), where + ".mixer"
            if kind == "parallel":
                mixer = ParallelConfig(_left(_get(m, "left", mw), mw + ".left"),
                                       _right(_get(m, "right", mw), mw + ".right", f"l{i}.mix.right.", shapes))
            elif kind == "lightning":
                mixer = _lightning(m, mw)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design (have: 'parallel', 'lightning')")
            layers.append(GataraxLayerConfig(kind, mixer, _feed_forward(entry.get("mlp"), where + ".mlp"), raw=entry))
        eps = _float(_get(d, "norm", "the model"), "eps", "norm")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cls(architecture=ARCHITECTURE, vocab_size=_int(d, "vocab", "the model"), hidden_size=_int(d, "width", "the model"),
                   norm_eps=eps, taps=_int(_get(d, "canon", "the model"), "taps", "canon"),
                   embedding_scale=_float(_get(d, "embedding", "the model"), "scale", "embedding"),
                   logit_scale=_float(d, "logit_scale", "the model"), layers=tuple(layers), raw=dict(d))

    def to_dict(self) -> dict:
        """The config.json form (the low ranks are written out)."""
        layers = []
        for L in self.layers:
            m, f = L.mixer, L.mlp
            if L.kind == "parallel":
                a, r = m.left, m.right
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "conv": a.conv}
                if a.window is not None:
                    left["mask"] = {"size": a.window}
                mixer = {"left": left, "right": {"heads": r.heads, "kv_heads": r.kv_heads, "dim": r.dim, "vdim": r.vdim, "conv": r.conv,
                                                 "decay_rank": r.decay_rank, "gate_rank": r.gate_rank}}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            mlp = None
            if isinstance(f, DenseMlpConfig):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff},
                       "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
            layers.append({"type": L.kind, "mixer": mixer, "mlp": mlp})
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                "canon": {"taps": self.taps}, "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
                "layers": layers}
