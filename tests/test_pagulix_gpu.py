"""The Pagulix decoder in the engine against the plain restatement (`plain_pagulix`): each mechanism's kernels alone,
then whole models: prompts whole, token by token, in portions down to two tokens, unequal batches, slots and pages used
again, keys at the edges of windows and of pages, far tokens, the first tokens of a sequence, long decoding, and greedy
generation through `Model.generate`."""
import math

import pytest
import torch

import pagulix_models as gm
import plain_pagulix as pp
from conftest import random_tokens, rel_err
from test_belizen_gpu import Streams, _Scratch, _run
from test_redodra_gpu import _drive, d, i32, make_ctx

# Worst row's max |a - b| / max |b| against the plain model in float64.  float32 runs: a kernel fault shows far above
# 1e-4.  bfloat16 runs keep bfloat16 activations between the kernels of a sublayer (the streams, the states, the norms,
# the router and the scores stay float32): rounding alone reaches 1e-2; a key too many or too few, a lost state, a missing
# sink or a wrong expert costs 0.2 and more.
TOL = {"float32": 1e-4, "bfloat16": 4e-2}


def _tol(name, dtype):
    """Model B's single recurrent heads are divided by a root mean square that is now and then small: rounding a sublayer's
    input to bfloat16 alone moves its logits by 0.05."""
    return 0.12 if name == "B" and dtype == "bfloat16" else TOL[dtype]


pytestmark = pytest.mark.gpu

DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16
PART_TOL = {F32: 3e-5, BF16: 3e-2}


def _cache(part, dtype, n_slots=2, max_tokens=1024, max_seq_len=512):
    from rust_inference_b200.cache.sequence_cache import SequenceCache
    return SequenceCache([part.cache_request()], max_tokens=max_tokens, max_seq_len=max_seq_len, dtype=dtype, device=DEV, n_slots=n_slots)


def _workspace():
    from rust_inference_b200.engine.context import Workspace
    return Workspace(DEV)


def _parts(layers, dtype, width, seed, eps=1e-5, edit=None, hot=1.0):
    """The parts (mixer, feed-forward) of the layers as the model's builder makes them, holding random tensors, and the same
    tensors in float64 for the plain functions."""
    from rust_inference_b200.parts.registry import lookup
    from rust_inference_b200.config.registry import config_from_dict, get_architecture
    cfg = gm.model(vocab=10, width=width, streams=2, factor=1.0, cap=1.0, eps=eps, layers=layers)
    W = {k: v.float() for k, v in pp.random_weights(cfg, seed, hot=hot).items()}
    if edit is not None:
        edit(W)
    spec = get_architecture("Pagulix").build_spec(config_from_dict(cfg))
    out = []
    for i, L in enumerate(spec.layers):
        made = []
        for role, category, prefix in (("mixer", "mixer", f"l{i}.mix."), ("feed_forward", "feed_forward", f"l{i}.mlp.")):
            ps = L.parts.get(role)
            if ps is None:
                made.append(None)
                continue
            part = lookup(category, ps.kind)(hidden_size=width, dtype=dtype, device=DEV, **ps.params)
            part.set_tensors({local: d(W[prefix + local], F32 if ts.role == "vector" else dtype) for local, ts in part.tensor_specs().items()})
            part.prepare(2048)
            made.append(part)
        out.append(made)
    return out, {k: v.double() for k, v in W.items()}


def _mixer(kind, m, dtype, width, seed, **kw):
    parts, W = _parts([gm.layer(kind, m)], dtype, width, seed, **kw)
    return parts[0][0], W


# ---------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("streams,width", [(1, 72), (2, 96), (2, 4096), (3, 130), (4, 516), (5, 64), (16, 33), (2, 4100), (3, 1030), (4, 8192)])
def test_streams_step(dtype, streams, width):
    """Writing a scaled result into all streams at once from the old ones, reading them for the next sublayer and its norm as one
    kernel, for one row, some and many; the accumulator is left zeroed; each half alone; chosen rows; a reading without norm."""
    from rust_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(streams * width)
    mix, write = torch.randn(streams, streams, generator=g), torch.randn(streams, generator=g)
    read = torch.randn(streams, generator=g)
    scale, norm = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    tol = 2e-5 if dtype == F32 else 8e-3
    for n in (1, 7, 400):
        x, y = torch.randn(n, streams, width, generator=g), torch.randn(n, width, generator=g)
        for scaled in (True, False):
            old = x.double().transpose(0, 1)
            new = pp.write_streams(old, mix.double(), write.double(), y.double() * (scale.double() if scaled else 1.0), 1.0)
            want = pp.rms_norm(pp.read_streams(new, read.double()), norm.double(), 1e-5)
            dx, dy, out = d(x.reshape(n, -1)).clone(), d(y).clone(), torch.empty(n, width, dtype=dtype, device=DEV)
            ops.streams_step(dx, streams, branch=dy, scale=d(scale) if scaled else None, mix=d(mix), write=d(write), read=d(read),
                             norm=d(norm), eps=1e-5, out=out)
            assert rel_err(dx, new.transpose(0, 1).reshape(n, -1)) < 3e-5
            assert rel_err(out, want) < tol
            assert float(dy.abs().max()) == 0.0
            alone, dy = d(x.reshape(n, -1)).clone(), d(y).clone()                      # written only: the same bits
            ops.streams_step(alone, streams, branch=dy, scale=d(scale) if scaled else None, mix=d(mix), write=d(write))
            assert torch.equal(alone, dx)
        rows = [n - 1, 0, n // 2]
        out = torch.empty(3, width, dtype=dtype, device=DEV)
        ops.streams_step(dx, streams, norm=d(norm), eps=1e-5, out=out, rows=i32(rows))  # the plain sum, chosen rows
        assert rel_err(out, pp.rms_norm(new.sum(0), norm.double(), 1e-5)[rows]) < tol
        out = torch.empty(n, width, dtype=F32, device=DEV)
        ops.streams_step(dx, streams, read=d(read), out=out)                           # no norm
        assert rel_err(out, pp.read_streams(new, read.double())) < 1e-5


def test_streams_step_refuses():
    from rust_inference_b200.kernels import ops
    x = torch.zeros(2, 34, device=DEV)
    with pytest.raises(ops.KernelError, match="at most"):
        ops.streams_step(x, 17, out=torch.zeros(2, 2, device=DEV))
    with pytest.raises(ops.KernelError, match="nothing to write"):
        ops.streams_step(x, 2)


@pytest.mark.parametrize("streams,width,top,n", [(2, 96, 1, 5), (3, 130, 4, 9), (2, 512, 6, 400), (4, 4096, 3, 7), (1, 64, 12, 300), (6, 72, 2, 3)])
def test_streams_step_sums_experts_rows(streams, width, top, n):
    """What routed experts leave (rows in the order of their lists, weights, a shared result, a factor) summed in the pass that
    writes the streams; rows in the pairs' own order; without a shared result."""
    from rust_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(streams * width)
    mix, write, read = torch.randn(streams, streams, generator=g), torch.randn(streams, generator=g), torch.randn(streams, generator=g)
    scale, norm = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    x, y = torch.randn(n, streams, width, generator=g), torch.randn(n * top, width, generator=g)
    weights, shared = torch.rand(n, top, generator=g), torch.randn(n, width, generator=g)
    order = torch.randperm(n * top, generator=g)
    for place, with_shared, factor in ((order, True, 0.7), (None, True, 1.0), (order, False, 1.0)):
        rows = (y[place] if place is not None else y).view(n, top, width).double()
        total = factor * ((weights.double()[:, :, None] * rows).sum(1) + (shared.double() if with_shared else 0.0))
        new = pp.write_streams(x.double().transpose(0, 1), mix.double(), write.double(), total * scale.double(), 1.0)
        dx, out = d(x.reshape(n, -1)).clone(), torch.empty(n, width, device=DEV)
        ops.streams_step(dx, streams, experts=dict(y=d(y), weights=d(weights), top=top, place=None if place is None else d(place.int()),
                                                   shared=d(shared) if with_shared else None, factor=factor),
                         scale=d(scale), mix=d(mix), write=d(write), read=d(read), norm=d(norm), eps=1e-5, out=out)
        assert rel_err(dx, new.transpose(0, 1).reshape(n, -1)) < 3e-5
        assert rel_err(out, pp.rms_norm(pp.read_streams(new, read.double()), norm.double(), 1e-5)) < 3e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,copies", [(72, 3), (30, 2), (512, 4)])
def test_embedding_into_several_streams(dtype, width, copies):
    from rust_inference_b200.kernels import ops
    table = torch.randn(11, width).to(dtype)
    ids = [3, 10, 0, 3]
    out = torch.empty(4, copies * width, device=DEV)
    ops.embed_gather(d(table), i32(ids), out)
    assert torch.equal(out.view(4, copies, width).cpu(), table[ids].float()[:, None].expand(4, copies, width))


def test_router_with_a_bias():
    """Ids and weights of the routing kernel against the plain router, the router's rows in one block per token and cut over
    several; a bias that overrules the logits, and the same with sigmoid scores."""
    from rust_inference_b200.kernels import ops
    for n, width, experts, top in ((1, 72, 6, 2), (9, 128, 16, 5), (40, 256, 72, 8), (700, 100, 32, 6), (3000, 64, 8, 8), (5, 64, 1, 1)):
        g = torch.Generator().manual_seed(n)
        x = torch.randn(n, width, generator=g)
        router, bias = torch.randn(experts, width, generator=g) / math.sqrt(width) * 2, torch.randn(experts, generator=g)
        bias[experts // 2] += 20.0
        ids, weights = pp.route(x.double(), router.double(), bias.double(), top)
        assert bool((ids == experts // 2).any(-1).all())
        s = torch.sigmoid(x.double() @ router.double().T + bias.double())
        sums = torch.empty(n, experts + 1, dtype=F32, device=DEV)
        tickets = torch.zeros(n, dtype=torch.int32, device=DEV)
        for split in ((1, 2, 5) if n < 296 else (1,)):
            kw = dict(top=top, bias=d(bias), split=split, split_sums=sums, split_count=tickets)
            got_ids, got_w = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
            ops.moe_route(d(x), d(router), None, got_ids, got_w, softmax=True, **kw)
            assert torch.equal(got_ids.cpu().long(), ids), (n, split)
            assert torch.allclose(got_w.cpu().double(), weights, rtol=2e-5, atol=1e-7), (n, split)
            ops.moe_route(d(x), d(router), None, got_ids, got_w, normalise=False, **kw)
            assert torch.allclose(got_w.cpu().double(), s.gather(1, got_ids.cpu().long()), rtol=2e-5, atol=1e-7)


@pytest.mark.parametrize("gated,stored", [(False, BF16), (True, BF16), (False, F32), (True, F32)])
def test_router_logits_as_a_product(gated, stored):
    """A long bfloat16 step forms the router's logits on the tensor cores, from as many bfloat16 matrices as its rows need (one
    where they are stored as bfloat16, three for float32 numbers): the same choices and weights as the float32 rows give, and
    the shared expert's gate with them.  Logits differ by float32 rounding only."""
    from rust_inference_b200.kernels import ops
    from rust_inference_b200.parts.registry import lookup
    width, n, experts, top = 200, 700, 11, 4
    g = torch.Generator().manual_seed(5)
    part = lookup("feed_forward", "routed_experts")(n_experts=experts, top=top, expert_size=16, shared_size=24, shared_gate=gated,
                                                    router_kind="softmax", router_bias=True, correction=False, hidden_size=width,
                                                    dtype=BF16, device=DEV)
    T = {k: (torch.randn(ts.shape, generator=g) / (math.sqrt(ts.shape[-1]) if len(ts.shape) > 1 else 1.0)) for k, ts in part.tensor_specs().items()}
    part.set_tensors({k: d(v.to(stored).float() if part.tensor_specs()[k].role == "vector" else v.to(BF16)) for k, v in T.items()})
    assert part.router_terms == (1 if stored == BF16 else 3)
    x = torch.randn(n, width, generator=g).to(BF16)
    ctx = _Scratch(_workspace(), BF16)
    cut = part.route_cut(d(x), ctx)
    z = x.double() @ part.router.double().cpu().T
    assert rel_err(cut["sums"][0].view(n, part.router_terms, -1)[:, :, :experts].sum(1), z) < 3e-6
    ids, weights = pp.route(x.double(), part.router.double().cpu(), part.router_bias.double().cpu(), top)
    got_ids, got_w, gate = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV), torch.empty(n, device=DEV)
    ops.moe_route(d(x), part.router, None, got_ids, got_w, top=top, softmax=True, bias=part.router_bias, gate_weight=part.shared_mix,
                  gate_out=gate if gated else None, **cut)
    assert torch.equal(got_ids.cpu().long(), ids)
    assert torch.allclose(got_w.cpu().double(), weights, rtol=2e-5, atol=1e-7)
    if gated:
        assert torch.allclose(gate.cpu().double(), torch.sigmoid(x.double() @ part.shared_mix.double().cpu()), rtol=1e-5)


# ---------------------------------------------------------------------------------------------------
# parts alone, outside an engine
# ---------------------------------------------------------------------------------------------------
# heads, kv heads, dim, vdim, rotated channels
ATTENTION_SIZES = [(4, 2, 16, 24, 8), (1, 1, 24, 24, 24), (5, 1, 12, 20, 4), (3, 3, 40, 9, 40), (4, 2, 64, 32, 32), (4, 1, 128, 64, 128), (6, 2, 128, 32, 96),
                   (4, 4, 64, 128, 16), (2, 1, 64, 64, 64), (6, 2, 128, 128, 48), (34, 2, 64, 32, 64), (2, 2, 96, 64, 96)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim,dims", ATTENTION_SIZES)
def test_attention_with_a_far_value_that_dwarfs_the_rest(dtype, heads, kv, dim, vdim, dims):
    """Rotation with stretched waves, weightless norms, values of their own size.  One position's value is made huge (channel 0
    of the input reaches the values only): before it the results are ordinary, from it on they show how much of its weight every
    query gives it, however far.  As one prompt, in portions and with the last tokens one by one."""
    width, n = 128, 330
    m = gm.attention(heads=heads, kv=kv, dim=dim, vdim=vdim, scale=0.6 / math.sqrt(dim), dims=dims, base=300.0, scaling=(4.0, 1.0, 4.0, 50.0))

    def edit(W):
        for name in ("q", "k"):
            W["l0.mix." + name][:, 0] = 0.0
    part, W = _mixer("attention", m, dtype, width, seed=dim + vdim, hot=1.5, edit=edit)
    cache, ws = _cache(part, dtype), _workspace()
    for big in (0, 63, 64, 130):
        x = (torch.randn(n, width, generator=torch.Generator().manual_seed(big)) * 0.3).to(dtype)
        x[:, 0] = 0.0
        x[big, 0] = 3e3
        want = pp.attention(x.double(), W, "l0.mix.", m, 1e-5, {})
        assert big == 0 or float(want[big].abs().max()) > 15 * float(want[big - 1].abs().max())
        for portions in ([n], [150, 1]):
            assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], (big, portions)
    assert rel_err(_drive(part, cache, x, [2, 1, 61, 3, 64, 7], dtype, ws), want) < PART_TOL[dtype]
    for first in (1, 2, 5):                                       # the first tokens of a sequence alone
        assert rel_err(_drive(part, cache, x[:first], [1], dtype, ws), want[:first]) < PART_TOL[dtype]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim,vdim,dims", [(64, 32, 64), (128, 64, 64), (128, 32, 128), (24, 16, 24), (64, 64, 32)])
def test_attention_finds_one_key_by_its_place(dtype, dim, vdim, dims):
    """All tokens are alike but one, whose key points the queries' way at that distance after the rotation only: a wrong angle,
    pairing or a norm taken elsewhere loses it.  Scores of up to sqrt(dim) * dim * scale."""
    width, n = 64, 200
    m = gm.attention(heads=2, kv=1, dim=dim, vdim=vdim, scale=1.0, dims=dims, base=20.0, scaling=(4.0, 0.5, 3.0, 60.0))
    part, W = _mixer("attention", m, dtype, width, seed=dim, hot=1.0)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(1)) * 0.5).to(dtype)
    want = pp.attention(x.double(), W, "l0.mix.", m, 1e-5, {})
    cache, ws = _cache(part, dtype), _workspace()
    tol = 1e-4 if dtype == F32 else 0.12                          # scores of 30 and more: a rounding of q and k moves them by 0.1
    for portions in ([n], [70, 1], [3]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < tol, portions


def _both(parts, caches, xs, portions, dtype, ws):
    """Two attention parts one after the other in every step, over one sequence: what each adds to a zeroed float32 stream."""
    n, width = xs[0].shape
    slots = [c.alloc_slot() for c in caches]
    got = [torch.zeros(n, width, device=DEV) for _ in parts]
    at, i = 0, 0
    while at < n:
        take = min(portions[min(i, len(portions) - 1)], n - at)
        extras = None
        for part, cache, slot, x, out in zip(parts, caches, slots, xs, got):
            ctx = make_ctx(cache, [slot], [at], [take], dtype, ws)
            if extras is not None:
                ctx.extras.update(extras)
            part.forward(d(x[at:at + take]), out[at:at + take], ctx, cache.layer(0), True)
            extras = ctx.extras
            cache.commit(slot, at + take)
        at, i = at + take, i + 1
    for c, s in zip(caches, slots):
        c.free_slot(s)
    return got


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 24), (2, 2, 64, 32), (4, 1, 128, 64), (3, 1, 12, 9)])
def test_values_blended_with_the_first_layer_s(dtype, heads, kv, dim, vdim):
    """Three layers whose heads may differ: the first keeps its own values, the others blend the first's in (not the blended
    ones of the layer before), each with its own number; whole prompts, portions, single tokens."""
    width, n = 96, 140
    ms = [gm.attention(heads=heads * k, kv=kv, dim=dim, vdim=vdim, scale=0.2, dims=dim if k == 1 else dim // 2, mix=True) for k in (1, 1, 2)]

    def edit(W):
        W["l1.mix.vmix"], W["l2.mix.vmix"] = torch.tensor(0.75), torch.tensor(-0.5)
        W["l0.mix.v"] *= 4.0
    made, W = _parts([gm.layer("attention", m) for m in ms], dtype, width, 3, edit=edit)
    parts = [p[0] for p in made]
    caches, ws = [_cache(p, dtype) for p in parts], _workspace()
    xs = [torch.randn(n, width, generator=torch.Generator().manual_seed(i)).to(dtype) for i in range(3)]
    shared = {}
    want = [pp.attention(x.double(), W, f"l{i}.mix.", m, 1e-5, shared) for i, (x, m) in enumerate(zip(xs, ms))]
    for portions in ([n], [70, 1, 2, 1], [2]):
        for got, w in zip(_both(parts, caches, xs, portions, dtype, ws), want):
            assert rel_err(got, w) < PART_TOL[dtype], portions
    with pytest.raises(RuntimeError, match="blended values"):
        _drive(parts[1], caches[1], xs[1], [n], dtype, ws)


# heads, dim, rotated part, vdim, rank, window
LATENT_SIZES = [(3, 12, 8, 20, 40, 20), (1, 24, 24, 24, 24, 1), (4, 32, 64, 64, 64, 70), (8, 64, 32, 32, 256, 129), (2, 16, 32, 16, 128, 64),
                (5, 9, 2, 7, 33, 65), (16, 32, 64, 32, 512, 40), (5, 48, 32, 40, 128, 33), (4, 40, 64, 24, 64, 200), (2, 128, 64, 128, 512, 100)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank,size", LATENT_SIZES)
def test_latent_window_edges_with_a_value_that_dwarfs_the_rest(dtype, heads, dim, rot_dim, vdim, rank, size):
    """Latent channel 0 comes from input channel 0 alone, makes no key and reaches the values with a large factor: one position
    stands out by orders of magnitude for the last query that sees it and is gone for the next one.  The position lies on
    both sides of a page border.  As one prompt, with the later tokens one by one, and in portions whose borders fall
    inside the window."""
    width, n, cut = 128, 330, 135
    m = gm.latent(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, rank=rank, scale=0.5 / math.sqrt(dim + rot_dim), base=200.0, size=size)

    def edit(W):
        p = "l0.mix."
        W[p + "q"][:, 0] = 0.0
        W[p + "dkv"][:, 0] = 0.0
        W[p + "dkv"][0] = 0.0
        W[p + "dkv"][0, 0] = 1.0
        W[p + "uk"][:, 0] = 0.0
        W[p + "uv"][:, 0] *= 1000.0
    part, W = _mixer("latent", m, dtype, width, seed=dim + size, hot=1.5, edit=edit)
    cache, ws = _cache(part, dtype), _workspace()
    for big in (0, 63, 64, 130):
        x = (torch.randn(n, width, generator=torch.Generator().manual_seed(big)) * 0.5).to(dtype)
        x[:, 0] = 0.0
        x[big, 0] = 20.0
        want = pp.latent_attention(x.double(), W, "l0.mix.", m, 1e-5)
        if big + size < n:
            assert float(want[big + size - 1].abs().max()) > 10 * float(want[big + size].abs().max())
        for portions in ([n], [cut, 1]):
            assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], (big, portions)
    assert rel_err(_drive(part, cache, x, [2, 1, 61, 3, 64, 7], dtype, ws), want) < PART_TOL[dtype]
    for first in (1, 2, 5):
        assert rel_err(_drive(part, cache, x[:first], [1], dtype, ws), want[:first]) < PART_TOL[dtype]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,rot_dim,rank,size", [(4, 32, 64, 70), (8, 64, 128, None), (3, 6, 40, 30), (2, 32, 512, None), (16, 64, 256, 20)])
def test_latent_sink_takes_what_the_keys_leave(dtype, heads, rot_dim, rank, size):
    """Sinks far below the scores, among them and far above: they take nothing, a share that depends on the number of keys
    seen, or everything.  Leaving one out, counting it per run of keys or scaling it changes a head's result by far more than
    rounding.  Whole prompts, portions and single tokens."""
    width, n = 96, 200
    m = gm.latent(heads=heads, dim=16, rot_dim=rot_dim, vdim=16, rank=rank, scale=0.05, size=size)

    def edit(W):
        W["l0.mix.sink"] = torch.tensor([-60.0, 3.0, 60.0, 5.0] * 4)[:heads].clone()
        W["l0.mix.uv"][:, 0] += 2.0                                # values that do not average out
        W["l0.mix.dkv"][0] = 0.0
        W["l0.mix.dkv"][0, 1] = 2.0
    part, W = _mixer("latent", m, dtype, width, seed=rank, edit=edit)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(4)) * 0.5).to(dtype)
    x[:, 1] = 2.0
    want = pp.latent_attention(x.double(), W, "l0.mix.", m, 1e-5)
    without = pp.latent_attention(x.double(), {**W, "l0.mix.sink": torch.full((heads,), -1e9, dtype=torch.float64)}, "l0.mix.", m, 1e-5)
    assert rel_err(without, want) > 0.2
    cache, ws = _cache(part, dtype), _workspace()
    for portions in ([n], [130, 1], [64, 2, 66, 5]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], portions


@pytest.mark.parametrize("rank,rot_dim,heads,size", [(64, 32, 5, 33), (128, 64, 16, 70), (256, 32, 8, 1), (512, 64, 20, 129), (512, 32, 3, None)])
def test_latent_attention_in_runs_of_keys(rank, rot_dim, heads, size):
    """The tensor-core kernel with window and sink, its keys in 1, 2, 3, 7 and 16 runs (some of them empty), single tokens and
    portions of unequal sequences: against the generic kernel on the same bfloat16 rows."""
    from rust_inference_b200.kernels import ops
    assert ops.latent_attention_mma_supports(rank, rot_dim, 64)
    wide = rank + rot_dim
    g = torch.Generator().manual_seed(rank + heads)
    sink = torch.randn(heads, generator=g) * 2
    starts_counts = [([300, 0, 63], [1, 1, 1]), ([100, 5, 128], [40, 1, 130])]
    from rust_inference_b200.cache.sequence_cache import KVRequest, SequenceCache
    for starts, counts in starts_counts:
        cache = SequenceCache([KVRequest(1, wide, size, rank, True)], max_tokens=1024, max_seq_len=512, dtype=BF16, device=DEV, n_slots=3)
        slots = [cache.alloc_slot() for _ in starts]
        ctx = make_ctx(cache, slots, starts, counts, BF16, _workspace())
        rows = cache.layer(0).k
        rows.copy_(torch.randn(rows.shape, generator=g))
        q = (torch.randn(sum(counts), heads * wide, generator=g) * 2).to(BF16).to(DEV)
        want = torch.empty(heads, sum(counts), rank, dtype=BF16, device=DEV)
        ops.attention_generic(q, q.shape[1], rows, rows, ctx.page_table, ctx.token_pos, ctx.token_seq, ctx.seq_slot, want,
                              n_tokens=len(q), n_heads=heads, n_kv_heads=1, head_dim=wide, page_size=64, scale=0.06, window=size or 0,
                              sink=d(sink), v_head_dim=rank, values_in_keys=True, head_major=True)
        for splits in (1, 2, 3, 7, 16):
            out = torch.full_like(want, float("nan"))
            po = torch.full((len(q) * heads * splits * rank,), float("nan"), device=DEV)
            pml = torch.full((len(q) * heads * splits * 2,), float("nan"), device=DEV)
            ops.latent_attention_mma(q, rows, ctx.page_table, ctx.seq_slot, ctx.seq_start, ctx.cu_seqlens, out, n_seqs=3, max_new=max(counts),
                                     n_heads=heads, rank=rank, rot_dim=rot_dim, scale=0.06, window=size or 0, sink=d(sink), n_splits=splits,
                                     part_o=po, part_ml=pml)
            assert rel_err(out.float().reshape(-1, rank), want.float().reshape(-1, rank)) < 3e-2, (starts, splits)


@pytest.mark.parametrize("kind", ["latent", "attention"])
def test_projections_split_over_k(kind):
    """A width whose small steps cut the projection over K into float32 accumulators: single tokens and portions that go that way
    against whole prompts that do not, and the accumulators zeroed again."""
    from rust_inference_b200.kernels import linear
    width, n = 1536, 300
    if kind == "latent":
        layers = [gm.layer("latent", gm.latent(heads=4, dim=32, rot_dim=16, vdim=24, rank=64, scale=0.15, size=50))]
    else:
        layers = [gm.layer("attention", gm.attention(heads=4, kv=2, dim=64, vdim=32, scale=0.125, dims=32, scaling=(4.0, 1.0, 4.0, 50.0), mix=True)),
                  gm.layer("attention", gm.attention(heads=2, kv=2, dim=24, vdim=32, scale=0.2, dims=24, mix=True))]
    made, W = _parts(layers, BF16, width, 6)
    parts = [p[0] for p in made]
    x = [torch.randn(n, width, generator=torch.Generator().manual_seed(3 + i)).to(BF16) for i in range(len(parts))]
    for part in parts:
        w = part.w_in if kind == "latent" else part.w_qkv
        assert linear.wants_split(d(x[0][:1]), w) and not linear.wants_split(d(x[0]), w)
    caches, ws, shared = [_cache(p, BF16) for p in parts], _workspace(), {}
    want = [pp.latent_attention(t.double(), W, f"l{i}.mix.", L["mixer"], 1e-5) if kind == "latent"
            else pp.attention(t.double(), W, f"l{i}.mix.", L["mixer"], 1e-5, shared) for i, (t, L) in enumerate(zip(x, layers))]
    for portions in ([n], [270, 1], [1, 2, 200, 30, 1], [64, 2]):
        for got, w in zip(_both(parts, caches, x, portions, BF16, ws), want):
            assert rel_err(got, w) < PART_TOL[BF16], portions
    acc = ws.get_zeroed("latent_proj_acc" if kind == "latent" else "qkv_acc", (256, 512), F32)
    assert float(acc.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim,conv", [(4, 2, 16, 24, 3), (1, 1, 40, 72, 1), (8, 4, 64, 48, 3), (2, 1, 128, 64, 2), (3, 3, 9, 7, 5)])
def test_delta_rule_alone(dtype, heads, kv, dim, vdim, conv):
    """With one decay per head and a silu gate: whole, in portions, token by token, in a slot another sequence has used."""
    width, n = 96, 150
    m = gm.delta(heads=heads, kv=kv, dim=dim, vdim=vdim, conv=conv)
    part, W = _mixer("delta", m, dtype, width, seed=dim + vdim, hot=1.5)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(conv)).to(dtype)
    want = pp.delta_rule(x.double(), W, "l0.mix.", m, 1e-5)
    cache, ws = _cache(part, dtype), _workspace()
    for portions in ([n], [1], [2], [70, 1, 1, 3, 33, 16, 17, 2]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], portions


def test_a_state_remembers_a_far_token():
    """With decays of almost 1 one large early input stays in the state: 300 tokens later the output still differs by far more
    than rounding, and the library agrees with the plain result on both, also token by token."""
    width, n = 64, 330
    m = gm.delta(heads=2, kv=1, dim=32, vdim=16, conv=2)

    def slow(W):
        W["l0.mix.A_log"].fill_(-9.0)
        W["l0.mix.dt_bias"].fill_(-1.0)
    part, W = _mixer("delta", m, F32, width, seed=5, edit=slow)
    a = torch.randn(n, width, generator=torch.Generator().manual_seed(9)) * 0.5
    b = a.clone()
    b[4] = b[4] * 8.0
    wa, wb = (pp.delta_rule(t.double(), W, "l0.mix.", m, 1e-5) for t in (a, b))
    assert float((wa[-1] - wb[-1]).abs().max()) > 1e-2 * float(wa[-1].abs().max())
    cache, ws = _cache(part, F32), _workspace()
    for x, want in ((a, wa), (b, wb)):
        for portions in ([n], [40, 1]):
            assert rel_err(_drive(part, cache, x, portions, F32, ws), want) < 1e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("experts,top,ff,shared", [(6, 3, 24, 40), (8, 2, 64, 96), (12, 5, 40, 8), (1, 1, 16, 24), (4, 4, 20, None), (9, 1, 96, 96), (8, 3, 32, 96),
                                                    (5, 2, 16, 128), (3, 2, 8, 80)])
def test_experts_as_a_part(dtype, experts, top, ff, shared):
    """The mixture against the plain one for 1, 7, 64, 65, 300 and 1,100 tokens, routed freely (both get the same rounded input): a
    shared expert as matrices of its own and, in small steps where it is a whole number of experts wide, as slices in the
    experts' lists; the tensors come back as they were."""
    width = 128
    mlp = gm.moe(experts=experts, top=top, ff=ff, shared=shared)
    parts, W = _parts([gm.layer("delta", gm.delta(heads=1, kv=1, dim=8, vdim=8, conv=1), mlp)], dtype, width, experts + top)
    part, ws = parts[0][1], _workspace()
    assert part.in_lists == (shared // ff if shared and shared % ff == 0 and shared // ff <= part.MOST_SLICES else 0)
    for name, t in part.get_tensors().items():
        assert torch.equal(t.double().cpu().reshape(W["l0.mlp." + name].shape), W["l0.mlp." + name]), name
    for n in (1, 7, 64, 65, 300, 1100):
        x = torch.randn(n, width, generator=torch.Generator().manual_seed(n)).to(dtype)
        got = torch.zeros(n, width, device=DEV)
        part.forward(d(x), got, _Scratch(ws, dtype))
        assert rel_err(got, pp.feed_forward(x.double(), W, "l0.mlp.", mlp)) < (3e-5 if dtype == F32 else 2e-2), n


# ---------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    made = {}

    def get(name, dtype="bfloat16", seed=0):
        pin = dtype == "bfloat16"                 # float32 runs route freely
        if (name, pin, seed) not in made:
            made[(name, pin, seed)] = gm.make(tmp_path_factory.mktemp("pagulix"), name, seed=seed, pin=pin)
        return made[(name, pin, seed)]
    return get


def _engine(model, dtype, **kw):
    from rust_inference_b200.engine.engine import Engine
    return Engine.from_pretrained(model.folder, dtype=dtype, max_tokens=kw.pop("max_tokens", 2048), n_slots=kw.pop("n_slots", 6), **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompt_layers_and_decoding(dtype, name, models):
    """A whole prompt (the sum of the streams after every layer too, and the same logits without looking), the same with its last
    tokens one by one (across the edges of windows and pages), and a slot used again: its states must start at zero, its
    pages hold old rows."""
    model = models(name, dtype)
    eng = _engine(model, dtype)
    tokens = random_tokens(230, model.cfg["vocab"], 1)
    streams = []
    want = model.plain_logits(tokens, streams=streams)
    tol = _tol(name, dtype)
    probe = Streams()
    s = eng.alloc_slot()
    got = eng.step([s], [tokens], "all", probe=probe)
    assert rel_err(got, want) < tol
    assert len(probe.seen) == len(streams) == len(model.cfg["layers"])
    for a, b in zip(probe.seen, streams):
        assert rel_err(a, b) < tol
    eng.free_slot(s)
    s1 = eng.alloc_slot()
    assert rel_err(eng.step([s1], [tokens], "all"), got.double().cpu()) < (1e-5 if dtype == "float32" else 2e-2)
    eng.free_slot(s1)
    s2 = eng.alloc_slot()
    assert s2 == s
    got = _run(eng, s2, tokens, [60, 1])
    assert rel_err(got, want) < tol
    eng.check_device_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions_of_several_sizes(dtype, name, models):
    model = models(name, dtype)
    eng = _engine(model, dtype)
    tokens = random_tokens(197, model.cfg["vocab"], 2)
    want = model.plain_logits(tokens)
    for portions in ([2], [1, 2, 3, 5, 7, 20, 19, 64, 2], [63, 1, 1, 66, 66], [64, 64, 69], [150, 47], [1]):
        s = eng.alloc_slot()
        assert rel_err(_run(eng, s, tokens, portions), want) < _tol(name, dtype), portions
        eng.free_slot(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_batch_against_each_alone(dtype, name, models):
    """Prompts of 1, 2, 70 and 160 tokens as one batch, then decoded together while the short ones leave; then a request in a
    freed slot (states that must start at zero) while the others still decode."""
    model = models(name, dtype)
    eng = _engine(model, dtype)
    vocab = model.cfg["vocab"]
    lens, extra = [1, 2, 70, 160], [3, 9, 30, 12]
    seqs = [random_tokens(n + e, vocab, 10 + i) for i, (n, e) in enumerate(zip(lens, extra))]
    want = [model.plain_logits(t) for t in seqs]
    slots = [eng.alloc_slot() for _ in seqs]
    out = eng.step(slots, [t[:n] for t, n in zip(seqs, lens)], "all").cpu()
    got, o = [], 0
    for n in lens:
        got.append([out[o:o + n]])
        o += n
    at = list(lens)
    second = None
    while any(a < len(t) for a, t in zip(at, seqs)):
        live = [b for b in range(len(seqs)) if at[b] < len(seqs[b])]
        out = eng.step([slots[b] for b in live], [[seqs[b][at[b]]] for b in live], "last").cpu()
        for i, b in enumerate(live):
            got[b].append(out[i:i + 1])
            at[b] += 1
            if at[b] == len(seqs[b]):
                eng.free_slot(slots[b])
        if second is None and len(live) < len(seqs):
            t2 = random_tokens(77, vocab, 99)
            s = eng.alloc_slot()
            second = rel_err(eng.step([s], [t2], "all"), model.plain_logits(t2))
            eng.free_slot(s)
    for b in range(len(seqs)):
        assert rel_err(torch.cat(got[b]), want[b]) < _tol(name, dtype), b
    assert second is not None and second < _tol(name, dtype)
    eng.check_device_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_and_short_requests_mixed_in_one_step(dtype, models):
    """A step that brings a portion of one request, single tokens of others and the start of another."""
    model = models("C", dtype)
    eng = _engine(model, dtype)
    vocab = model.cfg["vocab"]
    seqs = [random_tokens(n, vocab, 300 + n) for n in (150, 68, 80, 40)]
    want = [model.plain_logits(t) for t in seqs]
    slots = [eng.alloc_slot() for _ in range(3)]
    eng.step(slots, [seqs[0][:100], seqs[1][:66], seqs[2][:63]], "none")
    slots.append(eng.alloc_slot())
    out = eng.step(slots, [seqs[0][100:150], seqs[1][66:67], seqs[2][63:80], seqs[3]], "all").cpu()
    for part, w in zip(out.split([50, 1, 17, 40]), (want[0][100:], want[1][66:67], want[2][63:], want[3])):
        assert rel_err(part, w) < TOL[dtype]
    eng.check_device_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_captured_steps(dtype, name, models):
    """Three tokens of prompt, then 260 decode steps of a batch of two (captured steps), across four pages and past every
    window: logits of every step against the plain model."""
    model = models(name, dtype)
    eng = _engine(model, dtype)
    seqs = [random_tokens(263, model.cfg["vocab"], 21), random_tokens(263, model.cfg["vocab"], 22)]
    want = [model.plain_logits(t) for t in seqs]
    slots = [eng.alloc_slot(), eng.alloc_slot()]
    eng.step(slots, [t[:3] for t in seqs], "none")
    rows = [[], []]
    for p in range(3, 263):
        out = eng.step(slots, [[t[p]] for t in seqs], "last").cpu()
        rows[0].append(out[0:1])
        rows[1].append(out[1:2])
    assert eng.decode_graph(2) is not None and eng.decode_graph(2).graph is not None
    for b in range(2):
        assert rel_err(torch.cat(rows[b]), want[b][3:]) < TOL[dtype]
    eng.check_device_status()


def test_what_carries_a_far_token(tmp_path):
    """The first token lies outside every window of a late position: with latent layers alone the late logits do not depend on
    it; with a slow delta rule or an attention layer they do.  The engine agrees with the plain model in every case."""
    mlp = gm.moe(experts=3, top=2, ff=16, shared=16)
    lat = lambda: gm.layer("latent", gm.latent(heads=2, dim=16, rot_dim=8, vdim=16, rank=24, scale=0.2, size=9), mlp)
    att = lambda: gm.layer("attention", gm.attention(heads=2, kv=1, dim=16, vdim=16, scale=0.25, dims=16), mlp)
    rule = lambda: gm.layer("delta", gm.delta(heads=2, kv=1, dim=16, vdim=8, conv=3), mlp)

    def slow(W):
        for k in W:
            if k.endswith("A_log"):
                W[k].fill_(-8.0)
            if k.endswith("dt_bias"):
                W[k].fill_(-1.0)
    for name, layers, reaches in (("windows", [lat(), lat()], False), ("delta", [lat(), rule()], True), ("attention", [att(), lat()], True)):
        cfg = gm.model(vocab=97, width=64, streams=2, factor=0.6, cap=10.0, eps=1e-6, layers=layers)
        model = gm.make(tmp_path, name, cfg=cfg, edit=slow)
        eng = _engine(model, "float32")
        a = random_tokens(230, 97, 5)
        b = [(a[0] + 1) % 97] + a[1:]
        out = []
        for t in (a, b):
            s = eng.alloc_slot()
            got = _run(eng, s, t, [228, 1])
            eng.free_slot(s)
            assert rel_err(got, model.plain_logits(t)) < TOL["float32"], name
            out.append(got[-1])
        assert (float((out[0] - out[1]).abs().max()) > 1e-5) == reaches, name


def test_greedy_generation_through_the_api(models):
    """`Model.generate` (admission, prefill, captured decode steps, sampling on the device) against the plain model's greedy
    continuation, for prompts of unequal length; what a position costs in the cache."""
    from rust_inference_b200 import Model, SamplerConfig
    model = models("A", "float32")
    prompts = [random_tokens(5, model.cfg["vocab"], 31), random_tokens(40, model.cfg["vocab"], 32), [7]]
    n_new = 12
    m = Model.load(model.folder, dtype="float32", max_tokens_in_cache=1024)
    got = m.generate(prompts, n_new, SamplerConfig.plain(temperature=0.0), stop_ids=())
    for p, g in zip(prompts, got):
        assert list(g.tokens) == pp.greedy(model.cfg, model.weights, p, n_new)
    per = {"attention": lambda a: a["kv_heads"] * (a["dim"] + a["vdim"]), "latent_attention": lambda a: a["kv_rank"] + a["rot_dim"], "delta": lambda a: 0}
    assert m.memory()["cache_bytes_per_position"] == 4 * sum(per[L["type"]](L["mixer"]) for L in model.cfg["layers"])


@pytest.mark.parametrize("name", ["A", "B"])
def test_state_dict_round_trip(name, models):
    """The tensors come back apart under the file's names (but for the one that nothing reads)."""
    from rust_inference_b200 import Model
    model = models(name)
    m = Model.load(model.folder, dtype="float32", max_tokens_in_cache=512)
    sd = m.state_dict()
    assert set(model.weights) - set(sd) == ({"l0.mix.vmix"} if name == "A" else set()) and set(sd) <= set(model.weights)
    for k, v in sd.items():
        assert torch.equal(v.float().cpu().reshape(model.weights[k].shape), model.weights[k]), k


def test_trace_replay_picks_the_model_by_its_config(models, tmp_path):
    """`bin/trace_run` on a Pagulix folder: two requests start together, go on by one token and end at different steps; then
    a third request takes a slot given back."""
    import json
    import os
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    vocab = gm.CONFIGS["A"]["vocab"]
    a, b, c = (random_tokens(n, vocab, 40 + n) for n in (70, 9, 30))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[66]], "want": [0]}, {"id": "b", "tokens": [b[7]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[67]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[68]], "want": []}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": [a[69]], "want": [0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "c", "tokens": c, "want": [0, 29]}], "end": ["c"]}]
    for dtype in ("float32", "bfloat16"):
        model = models("A", dtype)
        out = tmp_path / ("out_" + dtype)
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", model.folder, "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(6)]
        wa, wb, wc = (model.plain_logits(t) for t in (a, b, c))
        read = lambda i, rows: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(rows, -1))
        assert not (out / "3.f32").exists()
        tol = TOL[dtype]
        assert rel_err(read(0, 3), torch.stack([wa[0], wa[65], wb[6]])) < tol
        assert rel_err(read(1, 1), wa[66:67]) < tol
        assert rel_err(read(2, 2), torch.stack([wa[67], wb[8]])) < tol
        assert rel_err(read(4, 1), wa[69:70]) < tol
        assert rel_err(read(5, 2), wc[[0, 29]]) < tol


def test_the_command_line_on_a_pagulix_folder(models):
    """`bin/gguf-infer` as a process: greedy ids from a model folder equal the plain model's."""
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    model = models("B", "float32")
    prompts = [random_tokens(n, model.cfg["vocab"], 70 + n) for n in (9, 1)]
    args = [sys.executable, os.path.join(root, "bin", "gguf-infer"), "--model", model.folder, "--temperature", "0",
            "--repetition-penalty", "1", "--max-tokens", "6", "--dtype", "float32", "--max-seq-len", "256", "--stop-ids", ""]
    for p in prompts:
        args += ["--prompt", ",".join(str(t) for t in p)]
    p = subprocess.run(args, capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [l for l in p.stdout.splitlines() if l.strip()]
    assert [[int(t) for t in l.split()] for l in lines] == [pp.greedy(model.cfg, model.weights, q, 6) for q in prompts]


@pytest.mark.parametrize("kind,m", [("attention", gm.attention(heads=4, kv=2, dim=64, vdim=32, scale=0.125, dims=64)),
                                    ("attention", gm.attention(heads=6, kv=2, dim=128, vdim=32, scale=0.08, dims=96)),
                                    ("attention", gm.attention(heads=4, kv=1, dim=128, vdim=64, scale=0.08, dims=64)),
                                    ("attention", gm.attention(heads=2, kv=2, dim=64, vdim=128, scale=0.125, dims=64)),
                                    ("latent", gm.latent(heads=5, dim=48, rot_dim=32, vdim=40, rank=128, scale=0.11, size=100))])
def test_tensor_core_kernels_take_the_forms(kind, m, monkeypatch):
    """bfloat16 runs of these sizes never reach the generic kernel: prompts, portions and single tokens, whose pages are cut into
    one run, several by a second kernel and several as a cluster."""
    from rust_inference_b200.kernels import attention, ops

    def refuse(*a, **k):
        raise AssertionError("the generic attention kernel was called")
    width, n = 128, 420
    part, W = _mixer(kind, m, BF16, width, seed=m["dim"], hot=1.5)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(3)) * 0.3).to(BF16)
    want = pp.attention(x.double(), W, "l0.mix.", m, 1e-5, {}) if kind == "attention" else pp.latent_attention(x.double(), W, "l0.mix.", m, 1e-5)
    cache, ws = _cache(part, BF16), _workspace()
    monkeypatch.setattr(ops, "attention_generic", refuse)
    for splits, decode in (("1", "auto"), ("3", "auto"), ("3", "tma"), (None, "auto")):
        monkeypatch.setattr(attention, "_DECODE", decode)
        if splits is None:
            monkeypatch.delenv("RI_B200_DECODE_SPLITS", raising=False)
        else:
            monkeypatch.setenv("RI_B200_DECODE_SPLITS", splits)
        assert rel_err(_drive(part, cache, x, [250, 130, 1], BF16, ws), want) < 3e-2
