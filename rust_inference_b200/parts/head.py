"""The output head: final norm, then logits = W h in float32, on the wanted rows only
(transformer.rs:89, :97).  The matrix is the embedding's when the model ties them: the same
storage, where the reference clones it (model.rs:221-226).  `scale`: logits = scale * W h (with the final norm where that can
take the factor, otherwise on the logits).  Of several parallel streams the head reads the sum.  `softcap` > 0: logits <- softcap * tanh(logits / softcap)."""
from __future__ import annotations

import torch

from ..kernels import linear, ops
from .base import Head
from .registry import lookup, register
from .spec import PartSpec, TensorSpec


@register("head", "linear_head")
class LinearHead(Head):
    def __init__(self, *, vocab_size: int, norm: PartSpec, tied: bool, weight_prefix: str | None = "lm_head.",
                 weight_name: str = "weight", softcap: float = 0.0, scale: float = 1.0, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        self.vocab_size = vocab_size
        self.wants_tie = bool(tied)
        self.softcap = float(softcap or 0.0)
        self.scale = float(scale)
        if self.softcap < 0:
            raise ValueError(f"a cap on the logits is not negative, found {softcap}")
        self.weight_prefix = weight_prefix
        self.weight_name = weight_name      # the matrix is the tensor weight_prefix + weight_name
        self.norm_prefix = norm.prefix
        self.norm = lookup("norm", norm.kind)(hidden_size=hidden_size, dtype=dtype, device=device, **norm.params)
        self.weight = None

    def tensor_specs(self):
        specs = {self.norm_prefix + local: ts for local, ts in self.norm.tensor_specs().items()}
        if not self.wants_tie:
            specs[self.weight_prefix + self.weight_name] = TensorSpec((self.vocab_size, self.hidden_size))
        return specs

    def set_tensors(self, tensors):
        n = len(self.norm_prefix)
        self.norm.set_tensors({name[n:]: t for name, t in tensors.items() if name.startswith(self.norm_prefix)
                               and name[n:] in self.norm.tensor_specs()})
        if not self.wants_tie:
            self.weight = linear.Weight(tensors[self.weight_prefix + self.weight_name])

    def get_tensors(self):
        out = {self.norm_prefix + local: t for local, t in self.norm.get_tensors().items()}
        if not self.wants_tie:
            out[self.weight_prefix + self.weight_name] = self.weight.t
        return out

    def tie(self, table):
        self.weight = linear.Weight(table)            # the same storage, no copy

    def prepare(self, max_positions):
        self.norm.prepare(max_positions)

    def matrix_bytes(self):
        return self.weight.t.numel() * self.weight.t.element_size()

    def _normed(self, residual, out, rows, factor=None, ctx=None):
        """out = the norm of the stream's (or the streams' summed) rows, times `factor` where one is given."""
        streams = residual.shape[1] // self.hidden_size
        if streams == 1:
            if factor is None:
                self.norm.forward(residual, out, rows=rows)
            else:
                self.norm.forward_times(factor, residual, out, rows=rows)
            return
        weight = getattr(self.norm, "factor", None)
        if weight is not None and factor is None:               # an RMS norm: sum and norm in one pass
            ops.streams_step(residual, streams, norm=weight, eps=self.norm.eps, out=out, rows=rows)
            return
        shape = tuple(out.shape)
        plain = (torch.empty(shape, dtype=torch.float32, device=out.device) if ctx is None
                 else ctx.buffer("head_streams", shape, torch.float32))
        ops.streams_step(residual, streams, out=plain, rows=rows)
        self._normed(plain, out, None, factor)

    def normalised(self, residual, rows):
        out = torch.empty((rows.numel(), self.hidden_size), dtype=self.dtype, device=residual.device)
        self._normed(residual, out, rows)
        return out

    def forward(self, residual, ctx, logits_out=None):
        normed = ctx.buffer("head_in", (ctx.n_logit_rows, self.hidden_size), self.dtype)
        with_norm = self.scale != 1.0 and hasattr(self.norm, "forward_times")
        self._normed(residual, normed, ctx.logit_rows, self.scale if with_norm else None, ctx)
        if logits_out is None:
            logits_out = torch.empty((ctx.n_logit_rows, self.vocab_size), dtype=torch.float32, device=residual.device)
        linear.logits(normed, self.weight, logits_out, ctx)
        if self.scale != 1.0 and not with_norm:
            ops.scale_(logits_out, self.scale)
        if self.softcap:
            ops.softcap_(logits_out, self.softcap)
        return logits_out
