"""The gated delta rule: a matrix state per head that is decayed, corrected towards the new value along the key, and
read by the query."""
from __future__ import annotations

import torch

from ..cache.sequence_cache import StateRequest
from ..kernels import linear, ops
from .base import Mixer
from .registry import register
from .spec import TensorSpec


@register("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    """q, k [n_kv_heads, head_dim] and v [n_heads, v_head_dim] are projections of the input that pass a short causal
    convolution per channel (taps [channels, K], the last column the current token's, no bias) and silu; q and k are
    then made unit vectors per head, x / sqrt(sum x^2 + 1e-6), q also times head_dim^(-1/2); head h reads the q/k head
    h // (n_heads / n_kv_heads).  With beta = sigmoid(W_b x) and g = exp(-exp(A_log) softplus(W_a x + dt_bias)), one of
    each per head:

        S <- g S;    u = beta (v - S^T k);    S <- S + k u^T;    o = S^T q            S: [head_dim, v_head_dim], float32

    so the read-out sees the token's own write.  Every head's o is RMS-normed over v_head_dim with one weight shared by
    the heads, multiplied by silu(W_g x) (heads side by side) and projected back.  State and the convolutions' last
    K - 1 inputs live in the slot's state area and are carried from step to step.  All projections run as one product
    with float32 results; everything up to the output projection is float32 in both precisions.  `out_scale`
    multiplies the mixer's result (in the norm).  `names` gives the tensors' names below the prefix.

    Further forms.  `decay_rank`: a decay per head and key channel, g = exp(-exp(A_log_h) softplus(W_a2 (W_a1 x) + dt_bias)),
    laid out head by head, from a low-rank map (`names`: decay_in [rank, hidden], decay_out [n_heads * head_dim, rank], in
    place of `a`; dt_bias then has n_heads * head_dim values): S <- diag(g) S.  `gate_rank`: the gate's pre-activation is
    W_g2 (W_g1 x) (`names`: gate_in, gate_out, in place of `gate`).  `gate_act`: "silu" or "sigmoid".  The two low-rank maps'
    inputs come out of the one product; a step of few tokens applies the maps in the preparing kernel, longer ones as
    products of their own (in bfloat16 runs the inputs enter as a rounded number and its rounded remainder, so that the decays
    keep 16 significant bits of them)."""

    _NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv1d.weight",
              "k_conv": "k_conv1d.weight", "v_conv": "v_conv1d.weight", "beta": "b_proj.weight", "a": "a_proj.weight",
              "dt_bias": "dt_bias", "A_log": "A_log", "gate": "g_proj.weight", "norm": "o_norm.weight", "o": "o_proj.weight",
              "decay_in": "a_proj.0.weight", "decay_out": "a_proj.1.weight", "gate_in": "g_proj.0.weight", "gate_out": "g_proj.1.weight"}

    def __init__(self, *, n_heads: int, n_kv_heads: int, head_dim: int, v_head_dim: int, conv: int, eps: float,
                 out_scale: float = 1.0, names: dict | None = None, decay_rank: int | None = None, gate_rank: int | None = None,
                 gate_act: str = "silu", hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        if n_kv_heads <= 0 or n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads are not a multiple of {n_kv_heads} query/key heads")
        if conv < 1:
            raise ValueError(f"a convolution has at least one tap, found {conv}")
        self.n_heads, self.n_kv_heads, self.head_dim, self.v_head_dim = int(n_heads), int(n_kv_heads), int(head_dim), int(v_head_dim)
        self.taps, self.eps, self.out_scale = int(conv), float(eps), float(out_scale)
        self.qk_dim, self.v_dim = self.n_kv_heads * self.head_dim, self.n_heads * self.v_head_dim
        self.conv_ch = 2 * self.qk_dim + self.v_dim
        self.decay_rank = None if decay_rank is None else int(decay_rank)
        self.gate_rank = None if gate_rank is None else int(gate_rank)
        for rank in (self.decay_rank, self.gate_rank):
            if rank is not None and rank < 1:
                raise ValueError(f"a low-rank map has a rank of at least one, found {rank}")
        if self.gate_rank is not None and self.decay_rank is None:
            raise ValueError("a low-rank gate comes with decays per key channel")
        if gate_act not in ("silu", "sigmoid"):
            raise ValueError(f"gated_delta_rule: unknown gate activation {gate_act!r}; known: silu, sigmoid")
        self.gate_act = gate_act
        # the projection's columns: q | k | v | gate (or its low-rank input) | beta | a (or the decays' low-rank input)
        self.gate_col = self.conv_ch
        self.beta_col = self.gate_col + (self.v_dim if self.gate_rank is None else self.gate_rank)
        self.a_col = self.beta_col + self.n_heads
        self.width = self.a_col + (self.n_heads if self.decay_rank is None else self.decay_rank)
        if self.decay_rank is not None:
            self.width = -(-self.width // 4) * 4               # rows of zeros up to a multiple of 16 bytes
        self.names = dict(self._NAMES, **(names or {}))
        self.w_in = self.w_o = self.w_conv = self.dt_bias = self.a_log = self.norm = None
        self.w_decay = self.w_gate = None                      # low-rank maps [channels, rank] ...
        self.w_decay_wide = self.w_gate_wide = None            # ... and as the products of long steps take them

    def tensor_specs(self):
        h, nm, K = self.hidden_size, self.names, self.taps
        specs = {
            nm["q"]: TensorSpec((self.qk_dim, h)), nm["k"]: TensorSpec((self.qk_dim, h)), nm["v"]: TensorSpec((self.v_dim, h)),
            nm["q_conv"]: TensorSpec((self.qk_dim, K), role="vector"), nm["k_conv"]: TensorSpec((self.qk_dim, K), role="vector"),
            nm["v_conv"]: TensorSpec((self.v_dim, K), role="vector"),
            nm["beta"]: TensorSpec((self.n_heads, h)), nm["a"]: TensorSpec((self.n_heads, h)),
            nm["dt_bias"]: TensorSpec((self.n_heads,), role="vector"), nm["A_log"]: TensorSpec((self.n_heads,), role="vector"),
            nm["gate"]: TensorSpec((self.v_dim, h)), nm["norm"]: TensorSpec((self.v_head_dim,), role="vector", init="ones"),
            nm["o"]: TensorSpec((h, self.v_dim)),
        }
        if self.decay_rank is not None:
            del specs[nm["a"]]
            channels = self.n_heads * self.head_dim
            specs.update({nm["decay_in"]: TensorSpec((self.decay_rank, h)), nm["decay_out"]: TensorSpec((channels, self.decay_rank)),
                          nm["dt_bias"]: TensorSpec((channels,), role="vector")})
        if self.gate_rank is not None:
            del specs[nm["gate"]]
            specs.update({nm["gate_in"]: TensorSpec((self.gate_rank, h)), nm["gate_out"]: TensorSpec((self.v_dim, self.gate_rank))})
        return specs

    @staticmethod
    def _wide(w):
        """A low-rank map for a product with `ops.low_rank_rows`: its rank padded to a multiple of 8, in bfloat16 twice side
        by side (for the inputs and for their remainders)."""
        rank = w.shape[1]
        padded = torch.zeros(w.shape[0], -(-rank // 8) * 8, dtype=w.dtype, device=w.device)
        padded[:, :rank] = w
        return linear.Weight(torch.cat([padded, padded], dim=1) if w.dtype == torch.bfloat16 else padded)

    def set_tensors(self, tensors):
        nm = self.names
        mats = [tensors[nm[n]] for n in ("q", "k", "v", "gate" if self.gate_rank is None else "gate_in", "beta",
                                         "a" if self.decay_rank is None else "decay_in")]
        rows = sum(m.shape[0] for m in mats)
        if rows < self.width:
            mats.append(torch.zeros(self.width - rows, self.hidden_size, dtype=mats[0].dtype, device=mats[0].device))
        self.w_in = linear.Weight(torch.cat(mats, dim=0))
        if self.decay_rank is not None:
            self.w_decay = tensors[nm["decay_out"]].contiguous()
            self.w_decay_wide = self._wide(self.w_decay)
        if self.gate_rank is not None:
            self.w_gate = tensors[nm["gate_out"]].contiguous()
            self.w_gate_wide = self._wide(self.w_gate)
        self.w_conv = torch.cat([tensors[nm["q_conv"]], tensors[nm["k_conv"]], tensors[nm["v_conv"]]], dim=0).contiguous()
        self.dt_bias, self.a_log = tensors[nm["dt_bias"]].contiguous(), tensors[nm["A_log"]].contiguous()
        self.norm = tensors[nm["norm"]].contiguous()
        self.w_o = linear.Weight(tensors[nm["o"]])

    def get_tensors(self):
        nm, qk, w, c = self.names, self.qk_dim, self.w_in.t, self.w_conv
        low_decay, low_gate = self.decay_rank is not None, self.gate_rank is not None
        a_rows = self.decay_rank if low_decay else self.n_heads
        out = {} if not low_decay else {nm["decay_out"]: self.w_decay}
        if low_gate:
            out[nm["gate_out"]] = self.w_gate
        return {**out, nm["q"]: w[:qk], nm["k"]: w[qk:2 * qk], nm["v"]: w[2 * qk:self.conv_ch],
                nm["gate_in" if low_gate else "gate"]: w[self.gate_col:self.beta_col], nm["beta"]: w[self.beta_col:self.a_col],
                nm["decay_in" if low_decay else "a"]: w[self.a_col:self.a_col + a_rows],
                nm["q_conv"]: c[:qk], nm["k_conv"]: c[qk:2 * qk], nm["v_conv"]: c[2 * qk:],
                nm["dt_bias"]: self.dt_bias, nm["A_log"]: self.a_log, nm["norm"]: self.norm, nm["o"]: self.w_o.t}

    def cache_request(self):
        return (StateRequest((self.n_heads, self.head_dim, self.v_head_dim), torch.float32),
                StateRequest((self.taps - 1, self.conv_ch), torch.float32))

    float32_projection = True       # the projection may come inside a wider matrix (`forward_projected`)

    def projection(self):
        return self.w_in

    def set_projection(self, w) -> None:
        self.w_in = w

    def forward(self, x, residual, ctx, cache_layer, writes_cache):
        z = ctx.buffer("scan_z", (x.shape[0], self.width), torch.float32)
        linear.logits(x, self.w_in, z, ctx)                            # float32 results in both precisions
        self.forward_projected(z, 0, residual, ctx, cache_layer, writes_cache)

    def forward_projected(self, z, col, residual, ctx, cache_layer, writes_cache):
        """`forward` from the projection: float32 [T, .], this part's columns from `col` on."""
        if not writes_cache:
            raise ValueError("a recurrent state has one writer: a layer cannot read another layer's state")
        matrix, carried = cache_layer.parts
        n, H, G = z.shape[0], self.n_heads, self.n_kv_heads
        u = ctx.buffer("scan_u", (n, -(-(self.conv_ch + 2 * H) // 4) * 4), torch.float32)
        common = dict(conv_col=col, conv_ch=self.conv_ch, taps=self.w_conv, conv_state=carried.state, unit_heads=2 * G,
                      unit_dim=self.head_dim, scaled_heads=G, unit_scale=self.head_dim ** -0.5, heads=H, step_col=col + self.beta_col,
                      a_log=self.a_log, dt_bias=self.dt_bias, out=u, cu_seqlens=ctx.cu_seqlens, token_seq=ctx.token_seq,
                      seq_slot=ctx.seq_slot, n_seqs=ctx.n_seqs, longest_run=ctx.max_new)
        gate, gate_col, decay = z, col + self.gate_col, None
        if self.decay_rank is None:
            ops.scan_prepare(z, conv_bias=None, decay_col=col + self.a_col, **common)
        else:
            decay = ctx.buffer("scan_decay", (n, H * self.head_dim), torch.float32)
            if self.gate_rank is not None:
                gate, gate_col = ctx.buffer("scan_gate", (n, self.v_dim), torch.float32), 0
            self._prepare_channels(z, col, decay, gate, n, ctx, common)
        o = ctx.buffer("scan_o", (n, self.v_dim), torch.float32)
        ops.state_scan(u, matrix.state, o, ctx.cu_seqlens, ctx.seq_slot, n_seqs=ctx.n_seqs, heads=H, groups=G,
                       dim=self.head_dim, vdim=self.v_head_dim, q_col=0, k_col=self.qk_dim, v_col=2 * self.qk_dim,
                       decay_col=self.conv_ch, step_col=self.conv_ch + H, delta=True, decay=decay, longest_run=ctx.max_new)
        normed = ctx.buffer("scan_normed", (n, self.v_dim), self.dtype)
        ops.gated_group_norm(o, gate, gate_col, self.norm, normed, groups=H, group_size=self.v_head_dim,
                             gate_first=False, gate_act=self.gate_act, eps=self.eps, out_scale=self.out_scale)
        linear.into_residual(normed, self.w_o, residual, ctx)

    def _low_rank_product(self, z, col, rank, wide, out, name, ctx):
        """out<float32> = (the map) z[:, col : col + rank]."""
        rows = ctx.buffer(name, (z.shape[0], wide.k), self.dtype)
        padded = wide.k // 2 if self.dtype == torch.bfloat16 else wide.k
        ops.low_rank_rows(z, col, rank, padded, rows)
        linear.logits(rows, wide, out, ctx)

    def _prepare_channels(self, z, col, decay, gate, n, ctx, common):
        """Convolved channels, steps, decays per key channel and the low-rank gate."""
        low_gate = self.gate_rank is not None
        if n <= ops.LOW_RANK_FORMED_TOKENS:
            gate_kw = dict(gate_w2=self.w_gate, gate_low_col=col + self.gate_col, gate_out=gate) if low_gate else {}
            ops.scan_prepare_channels(z, head_dim=self.head_dim, decay=decay, w2=self.w_decay, low_col=col + self.a_col, **gate_kw, **common)
            return
        self._low_rank_product(z, col + self.a_col, self.decay_rank, self.w_decay_wide, decay, "scan_low_decay", ctx)
        if low_gate:
            self._low_rank_product(z, col + self.gate_col, self.gate_rank, self.w_gate_wide, gate, "scan_low_gate", ctx)
        ops.scan_prepare_channels(z, head_dim=self.head_dim, decay=decay, raw=decay, **common)
