"""Linear attention whose state decays by a fixed number per head (the form known as lightning attention)."""
from __future__ import annotations

import torch

from ..cache.sequence_cache import StateRequest
from ..kernels import linear, ops
from .base import Mixer
from .registry import register
from .spec import TensorSpec


@register("mixer", "fixed_decay_linear_attention")
class FixedDecayLinearAttention(Mixer):
    """q = silu(Wq x) and k = silu(Wk x) [n_heads, head_dim], v = silu(Wv x) [n_heads, v_head_dim]; per head a state
    S [head_dim, v_head_dim] in float32, zero at the start of a sequence and carried in the slot's state area:

        S <- c_h S + k v^T          o = S^T q

    with a constant c_h per head (`decay`).  The heads' results, side by side, are RMS-normed together with one weight per
    channel, multiplied by sigmoid(Wg x) and projected back.  The four input projections run as one product with float32
    results, silu of the first three in its epilogue; state, norm and gate are float32 in both precisions.  The scan is the
    one of `selective_state_space` with decays that never change; long runs that would leave SMs idle are scanned in pieces
    side by side.  `out_scale` multiplies the mixer's result (in the norm).  `names` gives the tensors' names below the
    prefix."""

    _NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "gate": "g_proj.weight", "norm": "o_norm.weight",
              "o": "o_proj.weight"}

    def __init__(self, *, n_heads: int, head_dim: int, v_head_dim: int, decay, eps: float, out_scale: float = 1.0,
                 names: dict | None = None, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        self.n_heads, self.head_dim, self.v_head_dim = int(n_heads), int(head_dim), int(v_head_dim)
        self.decay = tuple(float(c) for c in decay)
        if len(self.decay) != self.n_heads:
            raise ValueError(f"{self.n_heads} heads need as many decays, found {len(self.decay)}")
        self.eps, self.out_scale = float(eps), float(out_scale)
        self.qk_dim, self.v_dim = self.n_heads * self.head_dim, self.n_heads * self.v_head_dim
        # the projection's columns: q | k | v | gate
        self.gate_col = 2 * self.qk_dim + self.v_dim
        self.width = self.gate_col + self.v_dim
        self.names = dict(self._NAMES, **(names or {}))
        self.w_in = self.w_o = self.norm = self.decays = self.activated = None

    def tensor_specs(self):
        h, nm = self.hidden_size, self.names
        return {nm["q"]: TensorSpec((self.qk_dim, h)), nm["k"]: TensorSpec((self.qk_dim, h)), nm["v"]: TensorSpec((self.v_dim, h)),
                nm["gate"]: TensorSpec((self.v_dim, h)), nm["norm"]: TensorSpec((self.v_dim,), role="vector", init="ones"),
                nm["o"]: TensorSpec((h, self.v_dim))}

    def set_tensors(self, tensors):
        nm = self.names
        self.w_in = linear.Weight(torch.cat([tensors[nm[n]] for n in ("q", "k", "v", "gate")], dim=0))
        self.w_o = linear.Weight(tensors[nm["o"]])
        self.norm = tensors[nm["norm"]].contiguous()
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=self.device)
        self.activated = torch.tensor([float(self.gate_col)], dtype=torch.float32, device=self.device)     # columns behind silu

    def get_tensors(self):
        nm, qk, w = self.names, self.qk_dim, self.w_in.t
        return {nm["q"]: w[:qk], nm["k"]: w[qk:2 * qk], nm["v"]: w[2 * qk:self.gate_col], nm["gate"]: w[self.gate_col:],
                nm["norm"]: self.norm, nm["o"]: self.w_o.t}

    def cache_request(self):
        return StateRequest((self.n_heads, self.head_dim, self.v_head_dim), torch.float32)

    def forward(self, x, residual, ctx, cache_layer, writes_cache):
        if not writes_cache:
            raise ValueError("a recurrent state has one writer: a layer cannot read another layer's state")
        n = x.shape[0]
        z = ctx.buffer("scan_z", (n, self.width), torch.float32)
        linear.logits(x, self.w_in, z, ctx, silu_cols=self.activated)
        o = ctx.buffer("scan_o", (n, self.v_dim), torch.float32)
        self.scan(z, cache_layer, o, ctx)
        normed = ctx.buffer("scan_normed", (n, self.v_dim), self.dtype)
        ops.gated_group_norm(o, z, self.gate_col, self.norm, normed, groups=1, group_size=self.v_dim, gate_first=False,
                             gate_act="sigmoid", eps=self.eps, out_scale=self.out_scale)
        linear.into_residual(normed, self.w_o, residual, ctx)

    def scan(self, z, cache_layer, o, ctx):
        """The recurrence over the step's tokens: o (float32 [T, heads * v_head_dim]) from the activated projection z."""
        H = self.n_heads
        piece, max_pieces = ops.scan_pieces(ctx.max_new, ctx.n_seqs * H * -(-self.v_head_dim // 16))
        pieces = {}
        if piece:                      # a long run of new tokens: its pieces side by side, from zero and again from their start states
            pieces = {"piece": piece, "max_pieces": max_pieces,
                      "piece_state": ctx.buffer("scan_piece_state", (ctx.n_seqs, max_pieces, H, self.head_dim, self.v_head_dim), torch.float32),
                      "piece_decay": ctx.buffer("scan_piece_decay", (ctx.n_seqs, max_pieces, H), torch.float32)}
        ops.state_scan(z, cache_layer.state, o, ctx.cu_seqlens, ctx.seq_slot, n_seqs=ctx.n_seqs, heads=H, groups=H,
                       dim=self.head_dim, vdim=self.v_head_dim, q_col=0, k_col=self.qk_dim, v_col=2 * self.qk_dim, decay_col=0,
                       step_col=0, delta=False, decay=self.decays, longest_run=ctx.max_new, **pieces)
