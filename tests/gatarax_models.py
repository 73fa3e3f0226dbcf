"""Small Gatarax configurations for the tests, random weights for them, and model folders made from both.

The configurations differ from one another in every size and constant and include values that make two sizes equal or
1: one kv head per query head and one for all, single heads, windows of one position, of less than a page, of more than
two pages and none, convolutions of one tap and of five, value heads narrower and wider than key heads, low ranks of 1 and
of no multiple of 4, one expert, as many experts chosen as there are, groups of one expert, one group and all groups
kept, decays of almost 1, of 0 and of exactly 1, layers without feed-forward, a width that is no multiple of 32."""
import json
import os

import torch

import plain_gatarax


def left(*, heads, kv, dim, vdim, scale, conv, size=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def right(*, heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(*, experts, top, ff, count=None, keep=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if count is not None:
        out["router"]["groups"] = {"count": count, "keep": keep}
    return out


def parallel(a, b, mlp):
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": mlp}


def lightning(*, heads, dim, vdim, decay, mlp):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def model(*, vocab, width, eps, taps, scale, logit_scale, layers):
    return {"architecture": "Gatarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": scale}, "logit_scale": logit_scale, "layers": layers}


CONFIGS = {
    "A": model(vocab=211, width=96, eps=1e-5, taps=4, scale=5.0, logit_scale=0.3, layers=[
        parallel(left(heads=4, kv=2, dim=16, vdim=24, scale=0.3, conv=3, size=20),
                 right(heads=4, kv=2, dim=16, vdim=24, conv=2), moe(experts=6, top=3, ff=40, count=3, keep=2)),
        lightning(heads=3, dim=16, vdim=8, decay=(0.5, 0.97, 0.999), mlp=None),
        parallel(left(heads=2, kv=2, dim=8, vdim=8, scale=0.5, conv=1, size=150),
                 right(heads=3, kv=1, dim=24, vdim=8, conv=5), dense(72)),
        lightning(heads=1, dim=40, vdim=24, decay=(0.9,), mlp=dense(40))]),
    "B": model(vocab=157, width=72, eps=1e-6, taps=1, scale=1.0, logit_scale=1.0, layers=[
        lightning(heads=2, dim=24, vdim=36, decay=(0.0, 1.0), mlp=moe(experts=1, top=1, ff=24)),
        parallel(left(heads=1, kv=1, dim=24, vdim=24, scale=0.2, conv=2, size=1),
                 right(heads=1, kv=1, dim=40, vdim=56, conv=1), dense(24)),
        parallel(left(heads=5, kv=1, dim=12, vdim=20, scale=0.25, conv=5, size=None),
                 right(heads=2, kv=2, dim=9, vdim=7, conv=3), None)]),
    # sizes the tensor-core kernels take: heads of 64 and 128, windows across pages
    "C": model(vocab=264, width=256, eps=1e-6, taps=2, scale=2.5, logit_scale=1.7, layers=[
        parallel(left(heads=4, kv=2, dim=64, vdim=64, scale=0.15, conv=4, size=70),
                 right(heads=4, kv=4, dim=64, vdim=128, conv=4), moe(experts=12, top=4, ff=64, count=4, keep=2)),
        lightning(heads=2, dim=128, vdim=64, decay=(0.8, 0.995), mlp=moe(experts=8, top=8, ff=32, count=8, keep=8)),
        parallel(left(heads=2, kv=1, dim=128, vdim=128, scale=0.09, conv=3, size=129),
                 right(heads=8, kv=2, dim=32, vdim=32, conv=2), dense(384))]),
}


def pin_routing(cfg, W):
    """Make the choice of experts the same for every token, with the routers' logits well apart, so that a rounding of
    the router's input cannot pick another expert: channel 0 of the stream is a constant that no layer touches, no
    convolution moves and the head does not read, and the routers read it with weights half a unit apart."""
    W["embed"][:, 0] = 3.0 / cfg["embedding"]["scale"]
    W["final.norm"][0] = -1.0
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        W[p + "norm1"][0] = 0.0
        for name in W:
            if name in (p + "mix.o", p + "mlp.down") or (name.startswith(p + "mlp.e") and name.endswith(".down")):
                W[name][0] = 0.0
            elif name in (p + "mix.left.out", p + "mix.right.out", p + "canon1", p + "canon2"):
                W[name][0] = 0.0
            elif name == p + "mlp.router":
                g = torch.Generator().manual_seed(i)
                W[name] = (0.1 * W[name].float()).to(W[name].dtype)
                W[name][:, 0] = 0.5 * torch.randperm(W[name].shape[0], generator=g).float().to(W[name].dtype)


class GataraxModel:
    def __init__(self, folder, cfg, weights):
        self.folder, self.cfg = folder, cfg
        self.weights = {k: v.float() for k, v in weights.items()}       # the stored bfloat16 values, widened

    def plain_logits(self, tokens, **kw):
        return plain_gatarax.forward(self.cfg, self.weights, tokens, **kw)


def make(tmp_path, name, seed=0, cfg=None, edit=None, pin=False, ranks=None, hot=1.0):
    """A model folder.  The low ranks stand in no configuration: the loader takes them from the tensors' shapes."""
    from rust_inference_b200.weights.safetensors_io import write_safetensors
    cfg = cfg or CONFIGS[name]
    weights = plain_gatarax.random_weights(cfg, seed, hot=hot, ranks=ranks)
    weights["embed"] = (weights["embed"].float() / max(cfg["embedding"]["scale"], 1.0)).to(torch.bfloat16)
    if pin:
        pin_routing(cfg, weights)
    if edit is not None:
        edit(weights)
    folder = str(tmp_path / f"gatarax_{name}_{seed}_{int(pin)}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights)
    return GataraxModel(folder, cfg, weights)
