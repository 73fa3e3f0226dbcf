"""Several mixers on the same input, their results summed with fixed factors."""
from __future__ import annotations

import torch

from ..kernels import linear, ops
from .base import Mixer
from .registry import lookup, register
from .spec import PartSpec, TensorSpec


@register("mixer", "parallel_mixers")
class ParallelMixers(Mixer):
    """residual += sum_m scale_m * mixer_m(x).  `members` lists (PartSpec, scale) pairs; a member's
    tensors sit below its spec's prefix, its factor is handed to it as `out_scale` (members apply it to
    their result in float32, before their output projection), and its cache is the member of the same
    place in the layer's composite cache request: an attention member keeps keys and values, a
    recurrent one a state, both in one cache layer.

    `member_norm` = {"eps": e, "weight_name": name}: every member's result is RMS-normed over the model width with a
    plain weight of its own (the tensor `name` below the member's prefix) before it is scaled and added:
    residual += sum_m scale_m * rmsnorm(mixer_m(x)) * w_m.  A member then writes into a zeroed float32 buffer of its
    own, and one kernel norms and adds all of them (with the output bias of a member that can hand it over).
    Members that all read their projections in float32 then have them as one product (their matrices lie one below the
    other): a step of few tokens cuts it over K into a zeroed accumulator, which the kernel that adds the results zeroes again."""

    def __init__(self, *, members, member_norm: dict | None = None, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        self.members = []
        self.member_norm = dict(member_norm) if member_norm else None
        if self.member_norm is not None and len(members) > 4:
            raise ValueError("parallel_mixers: at most four members are normed and added together")
        self.scales, self.norm_weights = [], []
        for spec, scale in members:
            if not isinstance(spec, PartSpec):
                raise TypeError("parallel_mixers: a member is a (PartSpec, scale) pair")
            inner_scale = 1.0 if self.member_norm is not None else float(scale)     # a norm would undo a factor before it
            part = lookup("mixer", spec.kind)(hidden_size=hidden_size, dtype=dtype, device=device,
                                              **dict(spec.params, out_scale=inner_scale))
            if self.member_norm is not None and getattr(part, "o_bias", False):
                part.hands_over_bias = True
            self.members.append((spec.prefix, part))
            self.scales.append(float(scale))
        self.w_in = None                 # the members' projections as one matrix, and where each begins
        self.cols = []
        if not self.members:
            raise ValueError("parallel_mixers: no members")
        self.graph_safe = all(getattr(p, "graph_safe", True) for _, p in self.members)

    def tensor_specs(self):
        out = {}
        for prefix, part in self.members:
            for local, ts in part.tensor_specs().items():
                if prefix + local in out:
                    raise ValueError(f"parallel_mixers: two members declare {prefix + local!r}")
                out[prefix + local] = ts
            if self.member_norm is not None:
                name = prefix + self.member_norm["weight_name"]
                if name in out:
                    raise ValueError(f"parallel_mixers: the member's norm weight {name!r} is a tensor of the member")
                out[name] = TensorSpec((self.hidden_size,), role="vector", init="ones")
        return out

    def set_tensors(self, tensors):
        for prefix, part in self.members:
            part.set_tensors({local: tensors[prefix + local] for local in part.tensor_specs()})
        if self.member_norm is not None:
            self.norm_weights = [tensors[prefix + self.member_norm["weight_name"]].contiguous() for prefix, _ in self.members]
            if all(getattr(part, "float32_projection", False) for _, part in self.members):
                mats = [part.projection().t for _, part in self.members]
                self.w_in = linear.Weight(torch.cat(mats, dim=0))
                self.cols, at = [], 0
                for (_, part), m in zip(self.members, mats):
                    part.set_projection(linear.Weight(self.w_in.t[at:at + m.shape[0]]))         # the same storage
                    self.cols.append(at)
                    at += m.shape[0]

    def get_tensors(self):
        out = {prefix + local: t for prefix, part in self.members for local, t in part.get_tensors().items()}
        if self.member_norm is not None:
            for (prefix, _), w in zip(self.members, self.norm_weights):
                out[prefix + self.member_norm["weight_name"]] = w
        return out

    def prepare(self, max_positions):
        for _, part in self.members:
            part.prepare(max_positions)

    def cache_request(self):
        return tuple(part.cache_request() for _, part in self.members)

    def forward(self, x, residual, ctx, cache_layer, writes_cache):
        if self.member_norm is None:
            for (_, part), sub in zip(self.members, cache_layer.parts):
                part.forward(x, residual, ctx, sub, writes_cache)
            return
        joined, z, cleared = [], None, None
        if self.w_in is not None:
            shape = (x.shape[0], self.w_in.n)
            if linear.wants_split(x, self.w_in):
                z = cleared = ctx.zeroed_buffer("members_z", shape, torch.float32)
                linear.accumulate_split(x, self.w_in, z, ctx)
            else:
                z = ctx.buffer("members_z", shape, torch.float32)
                linear.logits(x, self.w_in, z, ctx)
        for m, ((_, part), sub) in enumerate(zip(self.members, cache_layer.parts)):
            own = ctx.zeroed_buffer(f"member_result_{m}", tuple(residual.shape), torch.float32)
            if z is not None:
                part.forward_projected(z, self.cols[m], own, ctx, sub, writes_cache)
            else:
                part.forward(x, own, ctx, sub, writes_cache)
            joined.append((own, part.b_o if getattr(part, "hands_over_bias", False) else None, self.norm_weights[m], self.scales[m]))
        ops.normed_sum(joined, residual, self.member_norm["eps"], accumulate=True, clear=cleared)
