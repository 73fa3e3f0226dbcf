"""The Pagulix decoder as a `ModelSpec`.

Instead of one hidden stream there are several, all equal to the embedding's output at the start.  A sublayer (mixer, then
feed-forward) reads an RMS-normed weighted sum of them; its result, times a learned vector, is added to every stream with a
weight of its own while the streams are mixed with one another (`parallel_streams` with `stream_link` and `layer_scale`).  The
mixer is one of

* `latent_attention`: attention over a shared low-rank latent with interleaved rotation of the shared key part, a sliding
  window and a learned sink per head;
* `attention`: grouped-query attention with half-split rotation of a head's first channels, whose slow waves are stretched;
  q and k made unit-RMS per head; values blended with those of the first such layer (`value_mix`);
* `delta`: the gated delta rule with one decay per head.

The feed-forward is a mixture of gated experts, whose weights are the softmax over the chosen experts' biased logits, and a
shared expert that every token uses.  The head reads the sum of the streams, is tied to the embedding and caps its logits.

Tensor names: `embed`, `final.norm`, `l<i>.norm{1,2}`, `l<i>.ls{1,2}`, `l<i>.hc{1,2}.{in,out,mix}`,
`l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,o}`, `l<i>.mix.{q,k,v,vmix,o}`, `l<i>.mix.{q,k,v}{,.conv}`,
`l<i>.mix.{b,a,A_log,dt_bias,g,norm,o}`, `l<i>.mlp.router{,.b}`, `l<i>.mlp.{e<j>,shared}.{gate,up,down}`.
"""
from __future__ import annotations

from ..config.pagulix_config import ARCHITECTURE, PagulixConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, default_schedule

# the configuration gives no context length: positions are bounded by the cache a run is given
MAX_POSITIONS = 1 << 17

_LATENT_NAMES = {"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "sink": "sink", "o": "o"}
_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "value_mix": "vmix", "o": "o"}
_DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "beta": "b", "a": "a",
                "dt_bias": "dt_bias", "A_log": "A_log", "gate": "g", "norm": "norm", "o": "o"}
_EXPERT_NAMES = {"router": "router", "router_bias": "router.b", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down",
                 "shared_gate": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down"}


def _norm(prefix: str, eps: float) -> PartSpec:
    return PartSpec("rmsnorm", {"eps": eps, "weight_name": ""}, prefix=prefix)


def _mixer(L, eps: float, value_mix: str | None) -> PartSpec:
    m = L.mixer
    if L.kind == "latent_attention":
        position = PartSpec("rope", {"head_dim": m.rot_dim, "base": m.rot_base, "style": "interleaved", "exact_angles": True})
        return PartSpec("latent_attention", {
            "n_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim, "kv_rank": m.kv_rank, "eps": eps,
            "position": position, "scale": m.scale, "gated": False, "window": m.window, "sink": True, "names": _LATENT_NAMES},
            prefix="mix.")
    if L.kind == "attention":
        s = m.scaling
        waves = None if s is None else {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}
        position = PartSpec("rope", {"head_dim": m.dim, "base": m.rot_base, "style": "half", "rot_dims": m.rot_dims,
                                     "exact_angles": True, "wave_scaling": waves})
        return PartSpec("gqa_attention", {
            "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "qkv_bias": False,
            "position": position, "scale": m.scale, "qk_norm_eps": eps, "qk_norm_weights": False, "value_mix": value_mix,
            "names": _ATTENTION_NAMES}, prefix="mix.")
    return PartSpec("gated_delta_rule", {
        "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "conv": m.conv, "eps": eps,
        "names": _DELTA_NAMES}, prefix="mix.")


def _feed_forward(f) -> PartSpec:
    return PartSpec("routed_experts", {
        "n_experts": f.experts, "top": f.top, "expert_size": f.ff, "shared_size": f.shared_ff, "shared_gate": False,
        "router_kind": "softmax", "router_bias": True, "correction": False, "names": _EXPERT_NAMES}, prefix="mlp.")


def build_spec(cfg: PagulixConfig) -> ModelSpec:
    eps = cfg.norm_eps

    def around(q: int, role: str) -> dict:
        """What stands around sublayer q of a layer: its norm, its link to the streams, the vector on its result."""
        return {role + "_norm": _norm(f"norm{q}", eps),
                role + "_link": PartSpec("stream_link", {"streams": cfg.streams, "factor": cfg.residual_mult}, prefix=f"hc{q}."),
                role + "_scale": PartSpec("layer_scale", {"weight_name": ""}, prefix=f"ls{q}")}
    layers, unused, blended = [], [], False
    for i, L in enumerate(cfg.layers):
        value_mix = None
        if L.kind == "attention" and L.mixer.v_mix:
            value_mix = "mixed" if blended else "first"
            if not blended:
                unused.append(f"l{i}.mix.vmix")        # the first layer's values are the ones the others blend in
            blended = True
        parts = {"mixer": _mixer(L, eps, value_mix), **around(1, "mixer")}
        if L.mlp is not None:
            parts.update({"feed_forward": _feed_forward(L.mlp), **around(2, "feed_forward")})
        else:
            unused += [f"l{i}.norm2", f"l{i}.ls2", f"l{i}.hc2.*"]
        layers.append(LayerSpec(prefix=f"l{i}.", arrangement="parallel_streams", parts=parts))
    embedding = PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "weight_name": ""}, prefix="embed")
    head = PartSpec("linear_head", {"vocab_size": cfg.vocab_size, "norm": _norm("final.norm", eps), "tied": True,
                                    "weight_prefix": None, "softcap": cfg.logit_softcap})
    return ModelSpec(hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size, max_positions=MAX_POSITIONS, layers=tuple(layers),
                     schedule=default_schedule(len(layers)), embedding=embedding, head=head, streams=cfg.streams,
                     ignored_tensors=tuple(unused))


register_architecture(ARCHITECTURE, PagulixConfig.from_dict, build_spec, replace=True)
