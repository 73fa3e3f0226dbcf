"""What a sublayer reads, mixed with its last few inputs: a short causal convolution over time added to the input."""
from __future__ import annotations

from ..kernels import ops
from .base import Part
from .registry import register
from .spec import TensorSpec


@register("input_conv", "residual_short_conv")
class ResidualShortConv(Part):
    """h becomes h + conv(h), conv(h)_t = sum_j w[:, j] h_(t - taps + 1 + j) per channel, nothing before the sequence's
    start and no bias.  The tensor `weight_name` below the part's prefix is [hidden, taps], the last column the current
    token's.  The last taps - 1 values of h belong to the sequence's state; the arrangement that wires the part asks the cache
    for them (sublayers that read the same h share them) and runs the kernel, which does the norm in front and up to two
    convolutions in one pass (`run`)."""

    def __init__(self, *, taps: int, weight_name: str = "weight", hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        if taps < 1:
            raise ValueError(f"a convolution has at least one tap, found {taps}")
        self.taps, self.weight_name = int(taps), weight_name
        self.weight = None                      # [taps, hidden]: neighbouring channels side by side

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.hidden_size, self.taps), role="vector")}

    def set_tensors(self, tensors):
        self.weight = tensors[self.weight_name].t().contiguous()

    def get_tensors(self):
        return {self.weight_name: self.weight.t()}

    @staticmethod
    def run(stream, norm, first, second, carried, out_first, out_second, ctx) -> None:
        """out_first = h + conv_first(h) and, with `second`, out_second = h + conv_second(h), h = norm(stream).  An RMS norm
        (one with `factor` and `eps`) is part of the kernel; any other goes through a float32 buffer."""
        factor, eps = getattr(norm, "factor", None), getattr(norm, "eps", 0.0)
        x = stream
        if factor is None:
            x = ctx.buffer("input_conv_h", tuple(stream.shape), stream.dtype)
            norm.forward(stream, x)
        ops.input_conv(x, factor, eps, first.weight, second.weight if second is not None else None, carried, out_first,
                       out_second if second is not None else None, ctx.cu_seqlens, ctx.token_seq, ctx.seq_slot,
                       n_seqs=ctx.n_seqs, longest_run=ctx.max_new)
