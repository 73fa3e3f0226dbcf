"""Several parallel hidden streams instead of one: how a sublayer reads them and what it leaves in them."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Arrangement, Part
from .registry import register
from .spec import TensorSpec


@register("stream_link", "stream_link")
class StreamLink(Part):
    """One sublayer's link to `streams` parallel streams x_1 .. x_s.  The sublayer reads sum_s read[s] x_s; with y its result
    every stream becomes, all at once from the old ones, x_t <- sum_s mix[s, t] x_s + factor * write[t] * y (mix is indexed
    [from, to]).  `names`: read, write, mix below the part's prefix."""

    _NAMES = {"read": "in", "write": "out", "mix": "mix"}

    def __init__(self, *, streams: int, factor: float = 1.0, names: dict | None = None, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        if not 1 <= streams <= ops.MAX_STREAMS:
            raise ValueError(f"between 1 and {ops.MAX_STREAMS} parallel streams, found {streams}")
        self.streams, self.factor = int(streams), float(factor)
        self.names = dict(self._NAMES, **(names or {}))
        self.read = self.write = self.mix = None
        self.write_scaled = None                # factor * write

    def tensor_specs(self):
        s, nm = self.streams, self.names
        return {nm["read"]: TensorSpec((s,), role="vector", init="ones"), nm["write"]: TensorSpec((s,), role="vector", init="ones"),
                nm["mix"]: TensorSpec((s, s), role="vector", init="identity")}

    def set_tensors(self, tensors):
        nm = self.names
        self.read, self.write, self.mix = (tensors[nm[n]].contiguous() for n in ("read", "write", "mix"))
        self.write_scaled = (self.write * self.factor).contiguous()

    def get_tensors(self):
        nm = self.names
        return {nm["read"]: self.read, nm["write"]: self.write, nm["mix"]: self.mix}


@register("branch_scale", "layer_scale")
class LayerScale(Part):
    """A learned vector a sublayer's result is multiplied with, element by element, before it joins the stream.
    `weight_name` is the tensor's name below the part's prefix."""

    def __init__(self, *, weight_name: str = "weight", hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        self.weight_name = weight_name
        self.weight = None

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.hidden_size,), role="vector", init="ones")}

    def set_tensors(self, tensors):
        self.weight = tensors[self.weight_name].contiguous()

    def get_tensors(self):
        return {self.weight_name: self.weight}


class PendingWrite:
    """A sublayer's result that has not reached the streams yet (`result`: an accumulator as `branch`, or `experts`' rows; with
    its link and scale): the next sublayer's pass over the streams takes it along, or `apply` writes it."""

    def __init__(self, result: dict, link, scale):
        self.result, self.link, self.scale = result, link, scale

    def kwargs(self) -> dict:
        return dict(self.result, scale=None if self.scale is None else self.scale.weight, mix=self.link.mix,
                    write=self.link.write_scaled)

    def apply(self, stream) -> None:
        ops.streams_step(stream, self.link.streams, **self.kwargs())


@register("arrangement", "parallel_streams")
class ParallelStreams(Arrangement):
    """Mixer, then feed-forward, each reading norm(sum_s read[s] x_s) of the parallel streams x and writing back through its
    link (`StreamLink`), its result first multiplied by its scale where it has one.  A layer may have no feed-forward (and
    then no norm, link and scale for it).

    The stream tensor is [T, streams * hidden], a token's streams side by side.  A sublayer adds into a zeroed float32
    buffer; writing that into the streams, reading them for the next sublayer and the norm are one pass
    (`ops.streams_step`), also across layers; routed experts' rows are summed in that pass: what the layer's last sublayer leaves is taken along by the next layer, or
    written by the model where something else looks at the streams (`ctx.settle`)."""

    ROLES = {"mixer": "mixer", "feed_forward": "feed_forward", "mixer_norm": "norm", "feed_forward_norm": "norm",
             "mixer_link": "stream_link", "feed_forward_link": "stream_link", "mixer_scale": "branch_scale",
             "feed_forward_scale": "branch_scale"}
    OPTIONAL = ("feed_forward", "feed_forward_norm", "feed_forward_link", "feed_forward_scale", "mixer_scale")

    def __init__(self, **parts):
        super().__init__(**parts)
        absent = [getattr(self, "feed_forward" + role) is None for role in ("", "_norm", "_link")]
        if len(set(absent)) != 1 or (absent[0] and self.feed_forward_scale is not None):
            raise ValueError("parallel_streams: a feed-forward comes with its norm and link, and they with it")
        if self.feed_forward_link is not None and self.feed_forward_link.streams != self.mixer_link.streams:
            raise ValueError("parallel_streams: both sublayers of a layer are linked to the same streams")

    @staticmethod
    def _enter(stream, pending, link, norm, out, ctx):
        """Write what is pending, then out = norm(what `link` reads)."""
        kw = pending.kwargs() if pending is not None else {}
        factor = getattr(norm, "factor", None)
        if factor is not None:                  # an RMS norm is part of the pass
            ops.streams_step(stream, link.streams, read=link.read, norm=factor, eps=norm.eps, out=out, **kw)
            return
        plain = ctx.buffer("streams_read", tuple(out.shape), torch.float32)
        ops.streams_step(stream, link.streams, read=link.read, out=plain, **kw)
        norm.forward(plain, out)

    def forward(self, residual, ctx, cache_layer, writes_cache):
        shape = (residual.shape[0], residual.shape[1] // self.mixer_link.streams)
        normed = ctx.buffer("normed", shape, ctx.dtype)
        branch = ctx.zeroed_buffer("branch", shape, torch.float32)
        self._enter(residual, ctx.take_pending(), self.mixer_link, self.mixer_norm, normed, ctx)
        self.mixer.forward(normed, branch, ctx, cache_layer, writes_cache)
        pending = PendingWrite({"branch": branch}, self.mixer_link, self.mixer_scale)
        if self.feed_forward is not None:
            self._enter(residual, pending, self.feed_forward_link, self.feed_forward_norm, normed, ctx)
            experts = self.feed_forward.forward_unsummed(normed, ctx)
            if experts is None:
                self.feed_forward.forward(normed, branch, ctx)
            pending = PendingWrite({"branch": branch} if experts is None else {"experts": experts}, self.feed_forward_link, self.feed_forward_scale)
        ctx.leave_pending(pending)
