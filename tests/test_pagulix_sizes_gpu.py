"""Pagulix configurations drawn at random (seeded): every size and constant varies, including the ones the fixed test
models happen to make equal or 1; sizes the tensor-core attention kernels take and sizes only the generic one takes;
windows from one position to more than the prompt, and none; 1 to 6 streams; recurrent heads whose sizes are no multiple of 4;
any order of layers, with and without blended values.  Each model runs a prompt whole, in portions, its tail token by token
and in a batch of two unequal requests, in float32 (free routing) and bfloat16 (routing pinned), against the plain model."""
import random

import pytest
import torch

import pagulix_models as gm
from conftest import random_tokens, rel_err

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 6e-2}


def draw_config(seed: int) -> dict:
    rng = random.Random(8000 + seed)
    width = rng.choice([40, 64, 72, 96, 100, 128, 136])
    blend = (rng.choice([1, 2, 3]), rng.choice([8, 12, 32, 64]))      # the sizes values must have to be blended

    def mlp():
        if rng.random() < 0.15:
            return None
        experts = rng.choice([1, 2, 3, 5, 8])
        return gm.moe(experts=experts, top=rng.randint(1, min(4, experts)), ff=rng.choice([8, 16, 24, 40, 64]),
                      shared=rng.choice([None, 8, 24, 56, 64]))

    def attention():
        mix = rng.random() < 0.6
        kv, vdim = blend if mix else (rng.choice([1, 2, 3]), rng.choice([8, 9, 20, 32, 64, 128]))
        dim = rng.choice([8, 10, 16, 24, 40, 64, 64, 128, 128])
        scaling = None if rng.random() < 0.3 else (rng.uniform(2, 16), 1.0, rng.uniform(2, 6), rng.choice([16.0, 100.0, 1000.0]))
        return gm.layer("attention", gm.attention(
            heads=kv * rng.choice([1, 2, 4, 5]), kv=kv, dim=dim, vdim=vdim, scale=rng.uniform(0.5, 1.2) / dim ** 0.5,
            dims=rng.choice([dim, 2 * (dim // 4) or 2]), base=rng.choice([100.0, 10000.0, 1e6]), scaling=scaling, mix=mix), mlp())

    def latent():
        dim, rot = rng.choice([8, 12, 32, 40]), rng.choice([2, 6, 16, 32, 64])
        return gm.layer("latent", gm.latent(
            heads=rng.choice([1, 2, 3, 6]), dim=dim, rot_dim=rot, vdim=rng.choice([8, 9, 20, 32]), rank=rng.choice([16, 33, 64, 128]),
            scale=rng.uniform(0.5, 1.2) / (dim + rot) ** 0.5, base=rng.choice([100.0, 50000.0]),
            size=rng.choice([None, 1, 5, 33, 64, 65, 90, 128, 1000])), mlp())

    def delta():
        kv = rng.choice([1, 2, 3])
        return gm.layer("delta", gm.delta(heads=kv * rng.choice([1, 2, 3]), kv=kv, dim=rng.choice([14, 19, 32, 40, 64, 130]),
                                          vdim=rng.choice([12, 17, 32, 64, 100]), conv=rng.choice([1, 2, 3, 4, 5])), mlp())
    layers = [rng.choice([attention, latent, delta])() for _ in range(rng.choice([1, 2, 3, 4, 5]))]
    return gm.model(vocab=rng.choice([97, 160, 301]), width=width, streams=rng.choice([1, 2, 2, 3, 4, 6]), factor=rng.choice([0.3, 0.8, 1.0]),
                    cap=rng.choice([25.0, 60.0, 200.0]), eps=rng.choice([1e-5, 1e-6]), layers=layers)


@pytest.mark.parametrize("seed", list(range(16)))
def test_random_configuration(seed, tmp_path):
    from rust_inference_b200.engine.engine import Engine
    cfg = draw_config(seed)
    vocab = cfg["vocab"]
    a, b = random_tokens(150, vocab, seed), random_tokens(37, vocab, seed + 100)
    for dtype in ("float32", "bfloat16"):
        model = gm.make(tmp_path, f"r{seed}", seed=seed, cfg=cfg, pin=dtype == "bfloat16")
        want_a, want_b = model.plain_logits(a), model.plain_logits(b)
        eng = Engine.from_pretrained(model.folder, dtype=dtype, max_tokens=1024, n_slots=4)
        s = eng.alloc_slot()
        assert rel_err(eng.step([s], [a], "all"), want_a) < TOL[dtype], (seed, dtype, "whole", cfg)
        eng.free_slot(s)
        s = eng.alloc_slot()                    # the freed slot again, in portions down to two tokens
        rows, at = [], 0
        for take in (66, 2, 63, 2, 17):
            rows.append(eng.step([s], [a[at:at + take]], "all").cpu())
            at += take
        assert rel_err(torch.cat(rows), want_a) < TOL[dtype], (seed, dtype, "portions", cfg)
        eng.free_slot(s)
        sa, sb = eng.alloc_slot(), eng.alloc_slot()
        out = eng.step([sa, sb], [a[:131], b[:30]], "all").cpu()
        rows_a, rows_b = [out[:131]], [out[131:]]
        for p in range(7):
            out = eng.step([sa, sb], [[a[131 + p]], [b[30 + p]]], "last").cpu()
            rows_a.append(out[0:1])
            rows_b.append(out[1:2])
        eng.free_slot(sb)
        for p in range(138, 150):
            rows_a.append(eng.step([sa], [[a[p]]], "last").cpu())
        assert rel_err(torch.cat(rows_a), want_a) < TOL[dtype], (seed, dtype, "batch a", cfg)
        assert rel_err(torch.cat(rows_b), want_b) < TOL[dtype], (seed, dtype, "batch b", cfg)
        eng.check_device_status()
