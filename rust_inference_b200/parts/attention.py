"""Grouped-query attention over the cache (attention.rs:54-124)."""
from __future__ import annotations

import math

import torch

from ..cache.sequence_cache import KVRequest, StateRequest
from ..kernels import linear, ops, attention as attn_kernels
from .base import Mixer
from .registry import register, lookup
from .spec import TensorSpec, PartSpec


@register("mixer", "gqa_attention")
class GQAttention(Mixer):
    """q, k, v projections with optional biases (attention.rs:66-76), the position encoding
    on q and k fused with the cache write (:78-90), attention of every new token over the
    keys 0..position of its slot with scale 1/sqrt(head_dim) (:95-121), query head h reading
    kv head h / (heads / kv heads) (:37, :96), and the output projection without bias added
    onto the residual stream (:123, transformer.rs:38-39)."""

    # Beyond the dense decoder's form, as parameters: values of a head size of their own (`v_head_dim`),
    # a score scale other than 1/sqrt(head_dim) (`scale`), keys limited to the query's own block of
    # `chunk` positions counted from the start of the sequence, a factor on the mixer's result
    # (`out_scale`, applied to the attention's output in float32 before the output projection), and
    # the tensors' names below the part's prefix (`names`: q, k, v, o and, with biases, q_bias, ...).
    # `qk_norm_eps`: every q and k head is RMS-normalised before the rotation, with one weight of head_dim
    # values for the q heads and one for the k heads (`names`: q_norm, k_norm).  `values_from_keys`: there is
    # no value projection; a position's values are its keys as projected, before norm and rotation.
    # Forms of the score, the mask and the result (all off by default): `softcap` (scores become
    # softcap * tanh(score / softcap) after the scale); `distance_bias` (r1_h ln(1 + r2_h * distance) is taken off the
    # capped score, two learned numbers per head, `names`: r1, r2); `keep_first` (with a window: the first so many
    # positions of the sequence stay visible beyond it, at their true positions); `sink` (the softmax's denominator
    # also holds exp(sink_h), a learned number per head without key or value); `head_gate` (the head's result times
    # sigmoid(W_g x)_h, one more row per head in the projection, `names`: gate); `o_bias` (a bias on the output
    # projection, `names`: o_bias); `own_kv` False: the layer has no key and value projections and attends over the
    # cache of the layer the schedule gives it, with its own queries.  `out_gate`: the concatenated heads' result is
    # multiplied element by element with sigmoid(W_g x) before the output projection (one more row per value channel of
    # every head in the projection, `names`: out_gate).  `conv`: queries, keys and values each pass a short causal convolution
    # per channel right after the projection and its bias (so many taps, no activation; `names`: q_conv, k_conv, v_conv,
    # [channels, taps], the last column the current token's); the projection's last conv - 1 rows, biases included, are a
    # state of the sequence beside its keys and values.  `fixed_sink`: a sink that is the same number for every head and
    # no tensor.  `qk_norm_weights` False: the heads' norm has no weights (with a rotation that keeps lengths it is then
    # the same before and after it).  `value_mix`: the layer's values are blended with those of another layer of the same
    # step, v <- (1 - lambda) v + lambda v_first: "first" is the layer whose projected values are kept for the others (its own stay
    # as they are), "mixed" one that blends them in with its learned number lambda (`names`: value_mix); what is cached is blended.
    _NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight",
              "q_bias": "q_proj.bias", "k_bias": "k_proj.bias", "v_bias": "v_proj.bias",
              "q_norm": "q_norm.weight", "k_norm": "k_norm.weight", "o_bias": "o_proj.bias", "sink": "sinks",
              "gate": "gate_proj.weight", "r1": "distance_r1", "r2": "distance_r2", "out_gate": "out_gate_proj.weight",
              "q_conv": "q_conv1d.weight", "k_conv": "k_conv1d.weight", "v_conv": "v_conv1d.weight", "value_mix": "value_mix"}

    def __init__(self, *, n_heads: int, n_kv_heads: int, head_dim: int, qkv_bias: bool,
                 position: PartSpec, window: int | None = None, v_head_dim: int | None = None,
                 scale: float | None = None, chunk: int | None = None, out_scale: float = 1.0,
                 names: dict | None = None, qk_norm_eps: float | None = None, values_from_keys: bool = False,
                 softcap: float = 0.0, distance_bias: bool = False, keep_first: int = 0, sink: bool = False,
                 head_gate: bool = False, o_bias: bool = False, own_kv: bool = True, out_gate: bool = False,
                 conv: int | None = None, fixed_sink: float | None = None, qk_norm_weights: bool = True,
                 value_mix: str | None = None, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads are not a multiple of {n_kv_heads} kv heads")
        if chunk is not None and chunk <= 0:
            raise ValueError(f"a chunk holds at least one position, found {chunk}")
        self.n_heads, self.n_kv_heads, self.head_dim = n_heads, n_kv_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else int(v_head_dim)
        self.values_from_keys = bool(values_from_keys)
        if self.values_from_keys and self.v_head_dim != head_dim:
            raise ValueError(f"values taken from keys of size {head_dim} cannot have the size {self.v_head_dim}")
        if window is not None and window <= 0:
            raise ValueError(f"a window holds at least one position, found {window}")
        self.qk_norm_eps = None if qk_norm_eps is None else float(qk_norm_eps)
        self.qk_norm_weights = bool(qk_norm_weights)
        if value_mix not in (None, "first", "mixed"):
            raise ValueError(f"value_mix must be 'first' or 'mixed', found {value_mix!r}")
        if value_mix is not None and (values_from_keys or not own_kv or qkv_bias or conv is not None):
            raise ValueError("blended values go with value projections of the layer's own, without biases and convolutions")
        self.value_mix, self.value_lambda = value_mix, None
        self.q_dim, self.kv_dim = n_heads * head_dim, n_kv_heads * head_dim
        self.v_dim, self.o_dim = n_kv_heads * self.v_head_dim, n_heads * self.v_head_dim
        self.qkv_bias = bool(qkv_bias)
        if self.values_from_keys and self.qkv_bias:
            raise ValueError("values taken from keys and projection biases are not combined")
        self.q_norm = self.k_norm = None
        self.softcap, self.keep_first = float(softcap), int(keep_first or 0)
        self.distance_bias, self.sink, self.head_gate = bool(distance_bias), bool(sink), bool(head_gate)
        self.o_bias, self.own_kv, self.out_gate = bool(o_bias), bool(own_kv), bool(out_gate)
        if self.out_gate and self.head_gate:
            raise ValueError("a gate per head and a gate per channel are not combined")
        if self.softcap < 0 or self.keep_first < 0:
            raise ValueError(f"a score cap and a number of kept positions are not negative, found {softcap}, {keep_first}")
        if self.keep_first and window is None:
            raise ValueError("kept first positions go with a window")
        if not self.own_kv and (self.values_from_keys or self.qk_norm_eps is not None):
            raise ValueError("a layer without keys of its own has no key norm and no values taken from keys")
        # what only the general path (one projection, then the position encoding, then attention with these forms) does
        self.extended = bool(self.softcap or self.distance_bias or self.keep_first or self.sink or self.head_gate
                             or self.out_gate or not self.own_kv)
        self.conv = None if conv is None else int(conv)
        if self.conv is not None:
            if self.conv < 1:
                raise ValueError(f"a convolution has at least one tap, found {conv}")
            if (self.values_from_keys or self.qk_norm_eps is not None or self.head_gate or self.out_gate or not self.own_kv
                    or position.kind != "unrotated"):
                raise ValueError("convolved projections go without rotation, head norms, gates, values taken from keys and another layer's keys")
        if fixed_sink is not None and self.sink:
            raise ValueError("a learned sink and a fixed one are not combined")
        self.fixed_sink = None if fixed_sink is None else float(fixed_sink)
        self.extended = self.extended or self.fixed_sink is not None or self.conv is not None
        self.sinks = self.dist = self.b_o = None
        self.w_conv = None                      # [taps, channels]
        # a caller that adds the output projection's bias itself (with what it does next to the result) sets this
        self.hands_over_bias = False
        self.window = window
        self.chunk = chunk
        self.out_scale = float(out_scale)
        self.scale = 1.0 / math.sqrt(float(head_dim)) if scale is None else float(scale)
        self.names = dict(self._NAMES, **(names or {}))
        self.position = lookup("position", position.kind)(
            hidden_size=hidden_size, dtype=dtype, device=device, **position.params)
        self.w_qkv = self.b_qkv = self.w_o = None

    def tensor_specs(self):
        h, nm = self.hidden_size, self.names
        specs = {
            nm["q"]: TensorSpec((self.q_dim, h)),
            nm["k"]: TensorSpec((self.kv_dim, h)),
            nm["v"]: TensorSpec((self.v_dim, h)),
            nm["o"]: TensorSpec((h, self.o_dim)),
        }
        if self.values_from_keys:
            del specs[nm["v"]]
        if not self.own_kv:
            del specs[nm["k"]], specs[nm["v"]]
        if self.head_gate:
            specs[nm["gate"]] = TensorSpec((self.n_heads, h))
        if self.out_gate:
            specs[nm["out_gate"]] = TensorSpec((self.o_dim, h))
        if self.sink:
            specs[nm["sink"]] = TensorSpec((self.n_heads,), role="vector", init="zeros")
        if self.distance_bias:
            specs[nm["r1"]] = TensorSpec((self.n_heads,), role="vector", init="ones")
            specs[nm["r2"]] = TensorSpec((self.n_heads,), role="vector", init="ones")
        if self.o_bias:
            specs[nm["o_bias"]] = TensorSpec((h,), role="vector")
        if self.conv is not None:
            for name, rows in (("q_conv", self.q_dim), ("k_conv", self.kv_dim), ("v_conv", self.v_dim)):
                specs[nm[name]] = TensorSpec((rows, self.conv), role="vector")
        if self.value_mix == "mixed":
            specs[nm["value_mix"]] = TensorSpec((), role="vector", init="zeros")
        if self.qk_norm_eps is not None and self.qk_norm_weights:
            specs[nm["q_norm"]] = TensorSpec((self.head_dim,), role="vector", init="ones")
            specs[nm["k_norm"]] = TensorSpec((self.head_dim,), role="vector", init="ones")
        if self.qkv_bias:
            specs[nm["q_bias"]] = TensorSpec((self.q_dim,), role="vector")
            if self.own_kv:
                specs[nm["k_bias"]] = TensorSpec((self.kv_dim,), role="vector")
                specs[nm["v_bias"]] = TensorSpec((self.v_dim,), role="vector")
        return specs

    def set_tensors(self, tensors):
        nm = self.names
        # one matrix for the three projections: one pass over x
        mats = [tensors[nm["q"]]]
        if self.own_kv:
            mats += [tensors[nm["k"]]] + ([] if self.values_from_keys else [tensors[nm["v"]]])
        if self.head_gate or self.out_gate:
            # one more row per head (or per value channel of every head): the gates come out of the same product
            mats.append(tensors[nm["gate" if self.head_gate else "out_gate"]])
            rows = sum(m.shape[0] for m in mats)
            if rows % 8:                               # rows of zeros keep a token's row a multiple of 16 bytes, which the
                mats.append(torch.zeros(-rows % 8, mats[0].shape[1], dtype=mats[0].dtype, device=mats[0].device))   # tensor-core kernels want
        self.w_qkv = linear.Weight(torch.cat(mats, dim=0))
        if self.sink:
            self.sinks = tensors[nm["sink"]].contiguous()
        if self.fixed_sink is not None:
            self.sinks = torch.full((self.n_heads,), self.fixed_sink, dtype=torch.float32, device=self.device)
        if self.conv is not None:
            self.w_conv = torch.cat([tensors[nm[n]] for n in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()
        if self.distance_bias:
            self.dist = torch.stack([tensors[nm["r1"]], tensors[nm["r2"]]], dim=0).contiguous()
        if self.o_bias:
            self.b_o = tensors[nm["o_bias"]].contiguous()
            self.b_o_scaled = self.b_o if self.out_scale == 1.0 else self.b_o * self.out_scale
        if self.value_mix == "mixed":
            self.value_lambda = tensors[nm["value_mix"]].reshape(1).contiguous()
        if self.qk_norm_eps is not None and not self.qk_norm_weights:
            self.q_norm = self.k_norm = torch.ones(self.head_dim, dtype=torch.float32, device=self.device)
        elif self.qk_norm_eps is not None:
            self.q_norm, self.k_norm = tensors[nm["q_norm"]].contiguous(), tensors[nm["k_norm"]].contiguous()
        if self.qkv_bias:
            biases = [tensors[nm["q_bias"]]] + ([tensors[nm["k_bias"]], tensors[nm["v_bias"]]] if self.own_kv else [])
            self.b_qkv = torch.cat(biases, dim=0).contiguous()
            if self.b_qkv.numel() < self.w_qkv.n:      # the gates' rows, and the rows of zeros after them
                self.b_qkv = torch.cat([self.b_qkv, self.b_qkv.new_zeros(self.w_qkv.n - self.b_qkv.numel())]).contiguous()
        self.w_o = linear.Weight(tensors[nm["o"]])

    def get_tensors(self):
        q, kv, nm = self.q_dim, self.kv_dim, self.names
        w = self.w_qkv.t
        out = {nm["q"]: w[:q], nm["o"]: self.w_o.t}
        at = q
        if self.own_kv:
            out[nm["k"]] = w[q:q + kv]
            at = q + kv
            if not self.values_from_keys:
                out[nm["v"]] = w[at:at + self.v_dim]
                at += self.v_dim
        if self.head_gate:
            out[nm["gate"]] = w[at:at + self.n_heads]
        if self.out_gate:
            out[nm["out_gate"]] = w[at:at + self.o_dim]
        if self.sink:
            out[nm["sink"]] = self.sinks
        if self.distance_bias:
            out[nm["r1"]], out[nm["r2"]] = self.dist[0], self.dist[1]
        if self.o_bias:
            out[nm["o_bias"]] = self.b_o
        if self.value_mix == "mixed":
            out[nm["value_mix"]] = self.value_lambda.reshape(())
        if self.qk_norm_eps is not None and self.qk_norm_weights:
            out[nm["q_norm"]], out[nm["k_norm"]] = self.q_norm, self.k_norm
        if self.conv is not None:
            taps = self.w_conv.t()
            out[nm["q_conv"]], out[nm["k_conv"]], out[nm["v_conv"]] = taps[:q], taps[q:q + kv], taps[q + kv:]
        if self.qkv_bias:
            b = self.b_qkv
            out[nm["q_bias"]] = b[:q]
            if self.own_kv:
                out.update({nm["k_bias"]: b[q:q + kv], nm["v_bias"]: b[q + kv:q + kv + self.v_dim]})
        return out

    def prepare(self, max_positions):
        self.position.prepare(max_positions)

    def cache_request(self):
        keys = KVRequest(self.n_kv_heads, self.head_dim, self.window,
                         None if self.v_head_dim == self.head_dim else self.v_head_dim)
        if self.conv is None:
            return keys
        return keys, StateRequest((self.conv - 1, self.q_dim + self.kv_dim + self.v_dim), torch.float32)

    @property
    def float32_projection(self) -> bool:
        """True: the part reads its projection in float32 and can be handed it inside a wider matrix (`forward_projected`)."""
        return self.conv is not None

    def projection(self):
        return self.w_qkv

    def set_projection(self, w) -> None:
        self.w_qkv = w

    def _convolved(self, z, col, ctx, cache_layer, writes_cache):
        """The queries [T, heads * head_dim] behind the convolution of the projection (the columns of z from `col` on); keys
        and values go into the cache."""
        if not writes_cache:
            raise ValueError("a convolution's carried inputs have one writer: a layer cannot read another layer's")
        keys, carried = cache_layer.parts
        q = ctx.buffer("q_conv", (z.shape[0], self.q_dim), self.dtype)
        ops.conv_store(z, self.b_qkv, self.w_conv, carried.state, q, keys.k, keys.v, ctx.cu_seqlens, ctx.token_pos, ctx.token_seq,
                       ctx.seq_slot, ctx.page_table, n_seqs=ctx.n_seqs, n_kv_heads=self.n_kv_heads, head_dim=self.head_dim,
                       v_head_dim=self.v_head_dim, page_size=ctx.page_size, longest_run=ctx.max_new, z_col=col)
        return q, keys

    def forward_projected(self, z, col, residual, ctx, cache_layer, writes_cache):
        """`forward` from the projection: float32 [T, .], this part's columns from `col` on."""
        q, keys = self._convolved(z, col, ctx, cache_layer, writes_cache)
        self._attend(q, 0, residual, ctx, keys)

    def forward(self, x, residual, ctx, cache_layer, writes_cache):
        n = x.shape[0]
        if self.conv is not None:
            z = ctx.buffer("conv_z", (n, self.w_qkv.n), torch.float32)
            linear.logits(x, self.w_qkv, z, ctx)                       # float32 results in both precisions
            self.forward_projected(z, 0, residual, ctx, cache_layer, writes_cache)
            return
        # a layer that has key and value projections but is scheduled to read another layer's cache leaves its own unused
        kv_width = (self.kv_dim + (0 if self.values_from_keys else self.v_dim)) if self.own_kv else 0
        gate_col = self.q_dim + kv_width
        width = self.w_qkv.n                           # with gates: one more column per head, padded to a multiple of 8
        special = self.values_from_keys or self.qk_norm_eps is not None or self.value_mix is not None
        usual = (self.v_head_dim == self.head_dim and not getattr(self.position, "partial", False) and not special
                 and not self.extended)
        from_acc = getattr(self.position, "apply_and_store_from_accumulators", None) if usual else None
        if from_acc is not None and linear.wants_split(x, self.w_qkv):
            # a small step: the projection is split over K into float32 accumulators, and the
            # position encoding adds the bias, rotates and stores from there
            acc = ctx.zeroed_buffer("qkv_acc", (n, width), torch.float32)
            linear.accumulate_split(x, self.w_qkv, acc, ctx)
            qkv = ctx.buffer("q_rot", (n, self.q_dim), self.dtype)
            from_acc(acc, self.b_qkv, qkv, ctx, cache_layer, n_heads=self.n_heads, n_kv_heads=self.n_kv_heads,
                     head_dim=self.head_dim, write_kv=writes_cache)
        elif (special and not self.values_from_keys and not self.head_gate and not self.out_gate and writes_cache and self.own_kv
              and linear.wants_split(x, self.w_qkv) and hasattr(self.position, "apply_normed_and_store_from_accumulators")):
            # the same for heads that are normed, or whose values are blended
            acc = ctx.zeroed_buffer("qkv_acc", (n, width), torch.float32)
            linear.accumulate_split(x, self.w_qkv, acc, ctx)
            qkv = ctx.buffer("q_rot", (n, self.q_dim), self.dtype)
            keep = ctx.buffer("first_values", (n, self.v_dim), self.dtype) if self.value_mix == "first" else None
            self.position.apply_normed_and_store_from_accumulators(
                acc, self.b_qkv, qkv, ctx, cache_layer, n_heads=self.n_heads, n_kv_heads=self.n_kv_heads, head_dim=self.head_dim,
                q_weight=self.q_norm, k_weight=self.k_norm, eps=self.qk_norm_eps if self.qk_norm_eps is not None else 0.0,
                v_head_dim=self.v_head_dim, v_keep=keep, value_mix=self._blend(ctx, n, (keep, 0)))
        else:
            # values that later layers of the step blend in stay where they were projected: in a buffer that layers do not share
            qkv = ctx.buffer("qkv" if self.value_mix != "first" else "qkv_first_values", (n, width), self.dtype)
            linear.project(x, self.w_qkv, qkv, ctx, bias=self.b_qkv)
            extra = {} if usual else {"v_head_dim": self.v_head_dim}
            blend = self._blend(ctx, n, (qkv, self.q_dim + self.kv_dim))
            if blend is not None:
                extra["value_mix"] = blend
            if special:
                # norm of the heads, rotation and cache write as one kernel (the position encoding's)
                self.position.apply_normed_and_store(
                    qkv, ctx, cache_layer, n_heads=self.n_heads, n_kv_heads=self.n_kv_heads, head_dim=self.head_dim,
                    write_kv=writes_cache, q_weight=self.q_norm, k_weight=self.k_norm,
                    eps=self.qk_norm_eps if self.qk_norm_eps is not None else 0.0,
                    values_from_keys=self.values_from_keys, **extra)
            else:
                self.position.apply_and_store(qkv, ctx, cache_layer, n_heads=self.n_heads,
                                              n_kv_heads=self.n_kv_heads, head_dim=self.head_dim,
                                              write_kv=writes_cache and self.own_kv, **extra)
        self._attend(qkv, gate_col, residual, ctx, cache_layer)

    def _blend(self, ctx, n, own):
        """What the values are blended with, (lambda, rows, column), or None.  `own`: rows and column of the layer's own projected
        values, which later layers of the step read if this one is the first."""
        if self.value_mix == "first":
            ctx.extras["first_values"] = (*own, self.v_dim)
        if self.value_mix != "mixed":
            return None
        first = ctx.extras.get("first_values")
        if first is None or first[0].shape[0] != n or first[2] != self.v_dim:
            raise RuntimeError("blended values: no layer before this one has kept values of the same size in this step")
        return self.value_lambda, first[0], first[1]

    def _attend(self, qkv, gate_col, residual, ctx, cache_layer):
        """Attention over the cache, gates and the output projection; the queries are qkv's first columns."""
        mixed = ctx.buffer("attn_out", (qkv.shape[0], self.o_dim), self.dtype)
        attn_kernels.attention(qkv, cache_layer, mixed, ctx, n_heads=self.n_heads,
                               n_kv_heads=self.n_kv_heads, head_dim=self.head_dim, scale=self.scale,
                               window=self.window or 0, chunk=self.chunk or 0, v_head_dim=self.v_head_dim,
                               out_scale=1.0 if self.out_gate else self.out_scale, softcap=self.softcap,
                               keep_first=self.keep_first, sink=self.sinks, dist=self.dist,
                               gate=qkv[:, gate_col:gate_col + self.n_heads] if self.head_gate else None)
        if self.out_gate:
            # the gates of the projection's last columns, the mixer's factor with them (float32, one rounding)
            ops.sigmoid_gate_(mixed, qkv, gate_col, self.out_scale)
        linear.into_residual(mixed, self.w_o, residual, ctx)
        if self.o_bias and not self.hands_over_bias:
            ops.add_row_bias(residual, self.b_o_scaled)
