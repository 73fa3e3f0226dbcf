"""Registries of the parts a layer is assembled from, by kind.

A kind maps to a class; `LayerSpec` names kinds, never classes, and no part knows the
model it ends up in.  New parts register themselves here (also from outside the
package) and are then usable by any architecture's builder.

Interfaces (see `parts.base`):
  norm              Norm
  position encoding PositionEncoding
  mixer             Mixer
  feed-forward      FeedForward
  arrangement       Arrangement (how norms, mixer, feed-forward and residuals are wired; declares its roles)
  embedding         Embedding (token ids -> hidden stream)
  head              Head (hidden stream -> logits)
  depth             DepthMix (what a layer hands on, as a function of the results of all layers so far)
  stream_link       how a sublayer reads and writes several parallel streams (wired by an arrangement)
  branch_scale      a vector on a sublayer's result before it joins the stream (wired by an arrangement)
  input_conv        a short convolution in front of a sublayer (wired and run by an arrangement)
  stream            StreamStep (something that happens to the whole stream between layer runs the schedule names)
"""
from __future__ import annotations

_REGISTRIES: dict[str, dict] = {
    "norm": {}, "position": {}, "mixer": {}, "feed_forward": {}, "arrangement": {}, "embedding": {}, "head": {},
    "depth": {}, "stream": {}, "input_conv": {}, "stream_link": {}, "branch_scale": {},
}


def register(category: str, kind: str, *, replace: bool = False):
    """Class decorator: `@register("mixer", "gqa_attention")`."""
    if category not in _REGISTRIES:
        raise ValueError(f"unknown part category {category!r}; have {sorted(_REGISTRIES)}")

    def deco(cls):
        reg = _REGISTRIES[category]
        if kind in reg and not replace and reg[kind] is not cls:
            raise ValueError(f"{category} {kind!r} is already registered")
        reg[kind] = cls
        return cls
    return deco


def unregister(category: str, kind: str) -> None:
    _REGISTRIES[category].pop(kind, None)


def lookup(category: str, kind: str):
    _ensure_builtin()
    try:
        return _REGISTRIES[category][kind]
    except KeyError:
        raise KeyError(f"no {category} registered as {kind!r}; have {sorted(_REGISTRIES[category])}") from None


def kinds(category: str) -> list[str]:
    _ensure_builtin()
    return sorted(_REGISTRIES[category])


def _ensure_builtin() -> None:
    from . import norm, rope, attention, feed_forward, block, embedding, head  # noqa: F401
    from . import recurrence, parallel_mixer, routed_experts, latent_attention  # noqa: F401
    from . import depth, state_space, delta_rule  # noqa: F401
    from . import linear_attention, loop  # noqa: F401
    from . import input_conv, fixed_decay_attention  # noqa: F401
    from . import streams  # noqa: F401
