"""Gatarax configurations drawn at random (seeded): every size and constant varies, including the ones the fixed test
models happen to make equal or 1; head sizes of 64 and 128 with equal value heads send bfloat16 runs to the tensor-core
attention kernels, all others to the generic one; windows from one position to more than the prompt, and none; filters of
1 to 6 taps; recurrent heads whose sizes are no multiple of 4, low ranks from 1; 1 to 12 experts in groups of any size; any
order of layers.  Each model runs a prompt whole, in portions, its tail token by token and in a batch of two unequal
requests, in float32 (free routing) and bfloat16 (routing pinned), against the plain model."""
import random

import pytest
import torch

import gatarax_models as gm
from conftest import random_tokens, rel_err

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 6e-2}


def draw_config(seed: int) -> dict:
    rng = random.Random(7000 + seed)
    width = rng.choice([40, 64, 72, 96, 100, 128, 136])

    def mlp():
        r = rng.random()
        if r < 0.15:
            return None
        if r < 0.45:
            return gm.dense(rng.choice([8, 20, 24, 40, 72, 130]))
        count, size = rng.choice([1, 2, 3, 4]), rng.choice([1, 2, 3])
        keep = rng.randint(1, count)
        grouped = (count, keep) if count > 1 or rng.random() < 0.5 else (None, None)
        return gm.moe(experts=count * size, top=rng.randint(1, keep * size), ff=rng.choice([8, 16, 24, 40, 64]), count=grouped[0],
                      keep=grouped[1])

    def parallel():
        kv, rkv = rng.choice([1, 2, 3]), rng.choice([1, 2, 3])
        dim = rng.choice([8, 10, 16, 24, 40, 64, 64, 128])
        vdim = dim if dim in (64, 128) and rng.random() < 0.7 else rng.choice([8, 9, 12, 16, 40, 64])
        a = gm.left(heads=kv * rng.choice([1, 2, 4, 5]), kv=kv, dim=dim, vdim=vdim, scale=rng.uniform(0.05, 0.4),
                    conv=rng.choice([1, 2, 3, 4, 6]), size=rng.choice([None, 1, 5, 33, 64, 65, 90, 128, 1000]))
        b = gm.right(heads=rkv * rng.choice([1, 2, 3]), kv=rkv, dim=rng.choice([4, 9, 16, 40, 64, 130]),
                     vdim=rng.choice([6, 8, 17, 32, 64, 100]), conv=rng.choice([1, 2, 3, 4, 5]))
        return gm.parallel(a, b, mlp())

    def light():
        heads = rng.choice([1, 2, 3, 4])
        return gm.lightning(heads=heads, dim=rng.choice([4, 9, 16, 40, 64, 130]), vdim=rng.choice([6, 8, 17, 32, 64, 100]),
                            decay=[rng.choice([0.0, 0.5, 0.9, 0.99, 0.999, 1.0]) for _ in range(heads)], mlp=mlp())
    layers = [parallel() if rng.random() < 0.6 else light() for _ in range(rng.choice([1, 2, 3, 4]))]
    return gm.model(vocab=rng.choice([97, 160, 301]), width=width, eps=rng.choice([1e-5, 1e-6]), taps=rng.choice([1, 2, 3, 4, 6]),
                    scale=rng.choice([1.0, 5.0, 11.3]), logit_scale=rng.choice([0.1, 1.0, 3.7]), layers=layers)


@pytest.mark.parametrize("seed", list(range(14)))
def test_random_configuration(seed, tmp_path):
    from rust_inference_b200.engine.engine import Engine
    cfg = draw_config(seed)
    vocab = cfg["vocab"]
    rng = random.Random(seed)
    ranks = [(rng.choice([1, 3, 8, 16, 21]), rng.choice([1, 2, 8, 13])) for _ in cfg["layers"]]
    a, b = random_tokens(150, vocab, seed), random_tokens(37, vocab, seed + 100)
    for dtype in ("float32", "bfloat16"):
        model = gm.make(tmp_path, f"r{seed}", seed=seed, cfg=cfg, pin=dtype == "bfloat16", ranks=lambda i: ranks[i])
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
