"""The Gatarax decoder as a `ModelSpec`.

Every layer is x <- x + (mixer(h + conv_a(h)) + ff(h + conv_b(h))) with h = norm(x) (`parallel_shared_norm_conv`): one RMS
norm whose stored weight is an offset from one, and short causal convolutions of its output in front of both branches.
The mixer is one of

* `parallel`: attention without rotation over a sliding window, its biased projections behind short convolutions, a sink of
  score 0 in the softmax's denominator and a biased output projection (`gqa_attention` with `unrotated` positions, `conv`,
  `window`, `fixed_sink`, `o_bias`), beside the gated delta rule with a decay per key channel and an output gate from
  low-rank maps (`gated_delta_rule` with `decay_rank`, `gate_rank`, `gate_act`); each result is RMS-normed over the width and
  the two are averaged (`parallel_mixers` with `member_norm`);
* `lightning`: linear attention with a fixed decay per head (`fixed_decay_linear_attention`).

The feed-forward is W_down max(W_up x, 0)^2 (`dense_act`), a mixture of gated experts chosen by a softmax router among the
groups with the best single scores, whose plain scores are the weights (`routed_experts`), or absent.  The embedding is scaled
and tied to the head, which multiplies the logits by a number.

Tensor names: `embed`, `final.norm`, `l<i>.norm1`, `l<i>.canon{1,2}`, `l<i>.mix.{q,k,v,g,norm,o}`,
`l<i>.mix.left.{q,k,v}{,.b,.conv}`, `l<i>.mix.left.{o,o.b,out}`, `l<i>.mix.right.{q,k,v}{,.conv}`,
`l<i>.mix.right.{b,A_log,dt_bias,a1,a2,g1,g2,norm,o,out}`, `l<i>.mlp.{up,down}`, `l<i>.mlp.router`,
`l<i>.mlp.e<j>.{gate,up,down}`.
"""
from __future__ import annotations

from ..config.gatarax_config import ARCHITECTURE, DenseMlpConfig, GataraxConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, default_schedule

# the configuration gives no context length: positions are bounded by the cache a run is given
MAX_POSITIONS = 1 << 17

SINK_SCORE = 0.0             # the design's constant: the softmax's denominator has one more term exp(0)

_WINDOW_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
                 "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}
_DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "beta": "b",
                "decay_in": "a1", "decay_out": "a2", "dt_bias": "dt_bias", "A_log": "A_log", "gate_in": "g1", "gate_out": "g2",
                "norm": "norm", "o": "o"}
_LIGHTNING_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "norm": "norm", "o": "o"}
_DENSE_NAMES = {"up": "up", "down": "down"}
_EXPERT_NAMES = {"router": "router", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down"}


def _norm(prefix: str, eps: float) -> PartSpec:
    return PartSpec("rmsnorm", {"eps": eps, "unit_offset": True, "weight_name": ""}, prefix=prefix)


def _mixer(L, eps: float) -> PartSpec:
    m = L.mixer
    if L.kind == "lightning":
        return PartSpec("fixed_decay_linear_attention", {"n_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "decay": m.decay,
                                                         "eps": eps, "names": _LIGHTNING_NAMES}, prefix="mix.")
    a, r = m.left, m.right
    left = PartSpec("gqa_attention", {
        "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim, "qkv_bias": True, "o_bias": True,
        "position": PartSpec("unrotated", {}), "scale": a.scale, "window": a.window, "conv": a.conv, "fixed_sink": SINK_SCORE,
        "names": _WINDOW_NAMES}, prefix="left.")
    right = PartSpec("gated_delta_rule", {
        "n_heads": r.heads, "n_kv_heads": r.kv_heads, "head_dim": r.dim, "v_head_dim": r.vdim, "conv": r.conv, "eps": eps,
        "decay_rank": r.decay_rank, "gate_rank": r.gate_rank, "gate_act": "sigmoid", "names": _DELTA_NAMES}, prefix="right.")
    return PartSpec("parallel_mixers", {"members": ((left, 0.5), (right, 0.5)),
                                        "member_norm": {"eps": eps, "weight_name": "out"}}, prefix="mix.")


def _feed_forward(f) -> PartSpec:
    if isinstance(f, DenseMlpConfig):
        return PartSpec("dense_act", {"intermediate_size": f.ff, "activation": "relu_squared", "names": _DENSE_NAMES}, prefix="mlp.")
    return PartSpec("routed_experts", {
        "n_experts": f.experts, "top": f.top, "expert_size": f.ff, "n_groups": f.groups, "group_keep": f.keep,
        "group_score": "max", "router_kind": "softmax", "normalise": False, "correction": False, "names": _EXPERT_NAMES},
        prefix="mlp.")


def build_spec(cfg: GataraxConfig) -> ModelSpec:
    eps = cfg.norm_eps

    def conv(prefix):
        return PartSpec("residual_short_conv", {"taps": cfg.taps, "weight_name": ""}, prefix=prefix)
    layers, unused = [], []
    for i, L in enumerate(cfg.layers):
        parts = {"mixer": _mixer(L, eps), "norm": _norm("norm1", eps), "mixer_conv": conv("canon1")}
        if L.mlp is not None:
            parts["feed_forward"], parts["feed_forward_conv"] = _feed_forward(L.mlp), conv("canon2")
        else:
            unused.append(f"l{i}.canon2")              # nothing reads behind it
        layers.append(LayerSpec(prefix=f"l{i}.", arrangement="parallel_shared_norm_conv", parts=parts))
    embedding = PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "weight_name": "", "scale": cfg.embedding_scale},
                         prefix="embed")
    head = PartSpec("linear_head", {"vocab_size": cfg.vocab_size, "norm": _norm("final.norm", eps), "tied": True,
                                    "weight_prefix": None, "scale": cfg.logit_scale})
    return ModelSpec(hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size, max_positions=MAX_POSITIONS, layers=tuple(layers),
                     schedule=default_schedule(len(layers)), embedding=embedding, head=head, ignored_tensors=tuple(unused))


register_architecture(ARCHITECTURE, GataraxConfig.from_dict, build_spec, replace=True, reads_shapes=True)
