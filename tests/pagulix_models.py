"""Small Pagulix configurations for the tests, random weights for them, and model folders made from both.

The configurations differ from one another in every size and constant and include values that make two sizes equal or
1: one stream, two, three and five, one kv head per query head and one for all, single heads, windows of one position, of
less than a page, of more than two pages and none, value heads narrower and wider than key heads, whole and partly rotated
heads, rotations whose waves are kept, blended and stretched, blended values in no layer, in one and in several, filters of one
tap and of five, one expert, as many experts chosen as there are, shared experts of another size and none, layers without
feed-forward, a residual factor of 1, a width that is no multiple of 32."""
import json
import os

import torch

import plain_pagulix


def latent(*, heads, dim, rot_dim, vdim, rank, scale, base=10000.0, size=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def attention(*, heads, kv, dim, vdim, scale, dims, base=10000.0, scaling=None, mix=False):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "v_mix": mix}


def delta(*, heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def moe(*, experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(kind, mixer, mlp=None):
    return {"type": {"latent": "latent_attention"}.get(kind, kind), "mixer": mixer, "mlp": mlp}


def model(*, vocab, width, streams, factor, cap, eps, layers):
    return {"architecture": "Pagulix", "vocab": vocab, "width": width, "streams": streams, "residual_mult": factor,
            "logit_softcap": cap, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    "A": model(vocab=211, width=96, streams=3, factor=0.4, cap=40.0, eps=1e-5, layers=[
        layer("attention", attention(heads=4, kv=2, dim=16, vdim=24, scale=0.25, dims=8, base=500.0, scaling=(4.0, 1.0, 3.0, 100.0),
                                     mix=True), moe(experts=6, top=2, ff=40, shared=56)),
        layer("delta", delta(heads=4, kv=2, dim=16, vdim=24, conv=3), None),
        layer("latent", latent(heads=3, dim=12, rot_dim=8, vdim=20, rank=40, scale=0.3, size=20), moe(experts=5, top=3, ff=24, shared=24)),
        layer("attention", attention(heads=2, kv=2, dim=24, vdim=24, scale=0.2, dims=24, scaling=(8.0, 1.0, 4.0, 64.0), mix=True),
              moe(experts=3, top=1, ff=32))]),
    "B": model(vocab=157, width=72, streams=1, factor=1.0, cap=25.0, eps=1e-6, layers=[
        layer("latent", latent(heads=1, dim=24, rot_dim=24, vdim=24, rank=24, scale=0.2, size=1), moe(experts=1, top=1, ff=24, shared=8)),
        layer("delta", delta(heads=1, kv=1, dim=40, vdim=56, conv=1), moe(experts=4, top=4, ff=16, shared=40)),
        layer("attention", attention(heads=5, kv=1, dim=12, vdim=20, scale=0.3, dims=4), None),
        layer("delta", delta(heads=3, kv=3, dim=19, vdim=17, conv=5), moe(experts=2, top=1, ff=20, shared=12))]),
    # sizes the tensor-core kernels take: heads of 64 and 128, values of 32, 64 and 128, latents of 64 and 256, windows across pages
    "C": model(vocab=264, width=256, streams=2, factor=0.7, cap=60.0, eps=1e-6, layers=[
        layer("latent", latent(heads=4, dim=32, rot_dim=64, vdim=64, rank=64, scale=0.11, base=3000.0, size=70),
              moe(experts=12, top=4, ff=64, shared=128)),
        layer("attention", attention(heads=4, kv=2, dim=64, vdim=32, scale=0.125, dims=32, base=1e6, scaling=(8.0, 1.0, 4.0, 256.0)),
              moe(experts=8, top=2, ff=32, shared=32)),
        layer("attention", attention(heads=4, kv=1, dim=128, vdim=64, scale=0.08, dims=128, mix=True), moe(experts=4, top=3, ff=64, shared=64)),
        layer("delta", delta(heads=4, kv=2, dim=64, vdim=128, conv=4), moe(experts=4, top=2, ff=64, shared=64)),
        layer("latent", latent(heads=8, dim=64, rot_dim=32, vdim=32, rank=256, scale=0.1, size=129), None),
        layer("attention", attention(heads=2, kv=1, dim=64, vdim=64, scale=0.125, dims=64, mix=True), moe(experts=4, top=1, ff=96, shared=64))]),
}


def pin_routing(cfg, W):
    """Make the choice of experts the same for nearly every token, with the routers' logits well apart, so that a rounding of
    the router's input cannot pick another expert: the biases lie 1.2 apart and the matrices are small."""
    for name in W:
        if name.endswith("mlp.router"):
            W[name] = (0.08 * W[name].float()).to(W[name].dtype)
        elif name.endswith("mlp.router.b"):
            g = torch.Generator().manual_seed(len(name) + W[name].numel())
            W[name] = (1.2 * torch.randperm(W[name].numel(), generator=g).float()).to(W[name].dtype)


class PagulixModel:
    def __init__(self, folder, cfg, weights):
        self.folder, self.cfg = folder, cfg
        self.weights = {k: v.float() for k, v in weights.items()}       # the stored bfloat16 values, widened

    def plain_logits(self, tokens, **kw):
        return plain_pagulix.forward(self.cfg, self.weights, tokens, **kw)


def make(tmp_path, name, seed=0, cfg=None, edit=None, pin=False, hot=1.0):
    """A model folder."""
    from rust_inference_b200.weights.safetensors_io import write_safetensors
    cfg = cfg or CONFIGS[name]
    weights = plain_pagulix.random_weights(cfg, seed, hot=hot)
    if pin:
        pin_routing(cfg, weights)
    if edit is not None:
        edit(weights)
    folder = str(tmp_path / f"pagulix_{name}_{seed}_{int(pin)}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights)
    return PagulixModel(folder, cfg, weights)
